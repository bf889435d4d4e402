// Generalised delta rule (fp32 state and recurrence; bf16 or fp32 projections).  Per head, with
//   u = k / sqrt(k.k + 1e-6),  w = exp(-e^(-1/2) sigmoid(w0 + low-rank projection)),  a = sigmoid(a + bias):
//   S <- diag(w) S - (a u)(u^T S) + k v^T,   o = S^T r.
// The columns of S (value channels) never meet, and the output needs no second pass over the new state:
//   o = (w r)^T S_old - (r . a u)(u^T S_old) + (r . k) v
// so one sweep over S yields both dot products and a second one updates it.
//   hy_delta_tanh    tanh of the low-rank decay projection, in place, ahead of its second matrix
//   hy_delta_scan    prompt portions, token by token; state columns in registers
//   hy_delta_decode  one token per sequence; the state is read and written once
//   hy_delta_post    per head root-mean-square norm, gain, sigmoid gate -> the output projection's input
// State: [slot][head][key][value] fp32; a sequence at position 0 starts from zeros whatever its slot holds.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr float kDeltaUnit = 1e-6f;
constexpr float kDecayScale = 0.60653065971263342f;   // e^(-1/2)

template <typename T>
__global__ void __launch_bounds__(128)
hy_delta_tanh_kernel(T* __restrict__ proj, int ld, int off, int n, int rows) {
  const long t = (long)blockIdx.x * 128 + threadIdx.x;
  const int r = (int)(t / (n / 8)), i = (int)(t % (n / 8)) * 8;
  if (r >= rows) return;
  float f[8];
  load8(proj + (size_t)r * ld + off + i, f);
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = tanhf(f[j]);
  store8(proj + (size_t)r * ld + off + i, f);
}

// What a token brings to one head, in shared memory: unit key, decay, decay * r, removal (a u), k, v.
struct DeltaVecs {
  float *u, *w, *wr, *au, *k, *v;
};

// One warp turns the projections of a token into these vectors; returns (r . a u, r . k) in every lane.
template <typename T>
__device__ __forceinline__ float2 delta_token(const BbHyLayer& L, const T* row, const T* low, int h, const DeltaVecs& s) {
  const int lane = threadIdx.x & 31, D = L.p, o = h * L.pp;
  float kk = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float k = to_f(row[L.off_kk + o + d]);
    kk = fmaf(k, k, kk);
  }
  const float unit = 1.f / sqrtf(warp_sum(kk) + kDeltaUnit);
  float rau = 0.f, rk = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float k = to_f(row[L.off_kk + o + d]), r = to_f(row[L.off_r + o + d]), u = k * unit;
    const float w = expf(-kDecayScale * sigmoid_f(to_f(low[o + d]) + L.w0[o + d]));
    const float au = sigmoid_f(to_f(row[L.off_a + o + d]) + L.a_b[o + d]) * u;
    s.u[d] = u;
    s.w[d] = w;
    s.wr[d] = w * r;
    s.au[d] = au;
    s.k[d] = k;
    s.v[d] = to_f(row[L.off_vv + o + d]);
    rau = fmaf(r, au, rau);
    rk = fmaf(r, k, rk);
  }
  return make_float2(warp_sum(rau), warp_sum(rk));
}

// Any head size up to the shared memory: one block per (sequence, head), the state in shared memory, thread
// rows over keys and lanes over values.
constexpr int DS_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(DS_THREADS)
hy_delta_scan_any_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                         int ldl, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b, int seq0) {
  extern __shared__ __align__(16) float sm[];
  const int seq = seq0 + blockIdx.x, h = blockIdx.y, D = L.p;
  float* S = sm;                         // [D][D]
  float* vec = S + D * D;
  const DeltaVecs s{vec, vec + D, vec + 2 * D, vec + 3 * D, vec + 4 * D, vec + 5 * D};
  __shared__ float dots[2];
  float* red = vec + 6 * D;              // [rows][2][D]
  int lanes = 1;
  while (lanes < D && lanes < 32) lanes <<= 1;
  const int lane = threadIdx.x % lanes, kr = threadIdx.x / lanes, rows = DS_THREADS / lanes;
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.seq_pos0[seq] == 0;
  for (int i = threadIdx.x; i < D * D; i += DS_THREADS) S[i] = fresh ? 0.f : state[i];
  for (int r = r0; r < r1; ++r) {
    __syncthreads();
    if (threadIdx.x < 32) {
      const float2 d = delta_token<T>(L, proj + (size_t)r * ld, low + (size_t)r * ldl, h, s);
      if (threadIdx.x == 0) {
        dots[0] = d.x;
        dots[1] = d.y;
      }
    }
    __syncthreads();
    for (int j = lane; j < D; j += lanes) {
      float pu = 0.f, pr = 0.f;
      for (int i = kr; i < D; i += rows) {
        const float x = S[i * D + j];
        pu = fmaf(s.u[i], x, pu);
        pr = fmaf(s.wr[i], x, pr);
      }
      red[(kr * 2) * D + j] = pu;
      red[(kr * 2 + 1) * D + j] = pr;
    }
    __syncthreads();
    for (int j = lane; j < D; j += lanes) {
      float us = 0.f, os = 0.f;
      for (int q = 0; q < rows; ++q) {
        us += red[(q * 2) * D + j];
        os += red[(q * 2 + 1) * D + j];
      }
      const float v = s.v[j];
      if (kr == 0) y[(size_t)r * ldy + h * L.pp + j] = from_f<T>(fmaf(dots[1], v, fmaf(-dots[0], us, os)));
      for (int i = kr; i < D; i += rows)
        S[i * D + j] = fmaf(s.w[i], S[i * D + j], fmaf(s.k[i], v, -s.au[i] * us));
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < D * D; i += DS_THREADS) state[i] = S[i];
}

template <typename T>
__global__ void __launch_bounds__(128)
hy_delta_post_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ y, int ldy,
                     T* __restrict__ cat, int ldc, int rows, float eps) {
  const long w = ((long)blockIdx.x * 128 + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31, r = (int)(w / L.heads), h = (int)(w % L.heads), o = h * L.pp;
  if (r >= rows) return;
  const T* src = y + (size_t)r * ldy + o;
  float s = 0.f;
  for (int d = lane; d < L.p; d += 32) {
    const float f = to_f(src[d]);
    s = fmaf(f, f, s);
  }
  const float rstd = 1.f / sqrtf(warp_sum(s) / (float)L.p + eps);
  const T* g = proj + (size_t)r * ld + L.off_gg + o;
  T* dst = cat + (size_t)r * ldc + o;
  for (int d = lane; d < L.pp; d += 32)
    dst[d] = from_f<T>(d < L.p ? to_f(src[d]) * rstd * L.gnorm[o + d] * sigmoid_as<T>(to_f(g[d])) : 0.f);
}

template <typename T>
static int launch_scan(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int seq0, int n_seq, cudaStream_t s) {
  static PerDeviceOnce once;
  int lanes = 1;
  while (lanes < L.p && lanes < 32) lanes <<= 1;
  const size_t smem = 4ull * ((size_t)L.p * L.p + 6 * L.p + 2 * (DS_THREADS / lanes) * (size_t)L.p);
  if (smem > 220 * 1024) return BB_ESIZE;
  const cudaError_t e = ensure_dyn_smem(once, hy_delta_scan_any_kernel<T>, 220 * 1024);
  if (e != cudaSuccess) return (int)e;
  hy_delta_scan_any_kernel<T><<<dim3(n_seq, L.heads), DS_THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.y), w.ld_y, b, seq0);
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

BB_API int bb_hy_delta_tanh(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  const long t = (long)b->n * (L->wrp / 8);
  const int grid = (int)((t + 127) / 128);
  cudaStream_t s = (cudaStream_t)stream;
  if (c->dtype) hy_delta_tanh_kernel<float><<<grid, 128, 0, s>>>(static_cast<float*>(w->proj), w->ld_proj, L->off_w1, L->wrp, b->n);
  else hy_delta_tanh_kernel<__nv_bfloat16><<<grid, 128, 0, s>>>(static_cast<__nv_bfloat16*>(w->proj), w->ld_proj, L->off_w1, L->wrp, b->n);
  return (int)cudaGetLastError();
}

BB_API int bb_hy_delta_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->ns <= 0) return BB_OK;
  return c->dtype ? launch_scan<float>(*L, *w, *b, 0, b->ns, (cudaStream_t)stream)
                  : launch_scan<__nv_bfloat16>(*L, *w, *b, 0, b->ns, (cudaStream_t)stream);
}

BB_API int bb_hy_delta_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  const long t = (long)b->n * L->heads * 32;
  const int grid = (int)((t + 127) / 128);
  cudaStream_t s = (cudaStream_t)stream;
  if (c->dtype)
    hy_delta_post_kernel<float><<<grid, 128, 0, s>>>(*L, static_cast<const float*>(w->proj), w->ld_proj,
                                                     static_cast<const float*>(w->y), w->ld_y, static_cast<float*>(w->cat),
                                                     w->ld_cat, b->n, c->eps);
  else
    hy_delta_post_kernel<__nv_bfloat16><<<grid, 128, 0, s>>>(
        *L, static_cast<const __nv_bfloat16*>(w->proj), w->ld_proj, static_cast<const __nv_bfloat16*>(w->y), w->ld_y,
        static_cast<__nv_bfloat16*>(w->cat), w->ld_cat, b->n, c->eps);
  return (int)cudaGetLastError();
}

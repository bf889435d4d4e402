// Generalised delta rule (fp32 state and recurrence; bf16 or fp32 projections).  Per head, with
//   u = k / sqrt(k.k + 1e-6),  w = exp(-e^(-1/2) sigmoid(w0 + low-rank projection)),  a = sigmoid(a + bias):
//   S <- diag(w) S - (a u)(u^T S) + k v^T,   o = S^T r.
// The columns of S (value channels) never meet, and the output needs no second pass over the new state:
//   o = (w r)^T S_old - (r . a u)(u^T S_old) + (r . k) v
// so one sweep over S yields both dot products and a second one updates it.
//   hy_delta_tanh    tanh of the low-rank decay projection, in place, ahead of its second matrix
//   hy_delta_scan    prompt portions, token by token; the state in registers, its columns spread over warps and
//                    blocks, while other warps prepare the next tokens' vectors (bf16, heads up to 128)
//   hy_delta_scan_any  the same with the state in shared memory: fp32, and other head sizes
//   hy_delta_decode  one token per sequence: the state is read and written once, norm and gate included
//   hy_delta_post    per head root-mean-square norm, gain, sigmoid gate -> the output projection's input
// In fp32 the decay is applied as S + (w - 1) S: where w is close to one its rounding to 32 bits would change
// the rate of a slow decay by 2^-25 / (1 - w).
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

// What a token brings to one head, in shared memory: unit key, decay * r, decay (fp32: less one), k,
// removal (a u), v.
struct DeltaVecs {
  float *u, *wr, *w, *k, *au, *v;
  __device__ static DeltaVecs at(float* p, int n) { return {p, p + n, p + 2 * n, p + 3 * n, p + 4 * n, p + 5 * n}; }
};

// One warp turns the projections of a token into these vectors (zeros from D to DP); returns (r . a u, r . k)
// in every lane.
template <typename T>
__device__ __forceinline__ float2 delta_token(const BbHyLayer& L, const T* row, const T* low, int h, const DeltaVecs& s, int DP) {
  const int lane = threadIdx.x & 31, D = L.p, o = h * L.pp;
  float kk = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float k = to_f(row[L.off_kk + o + d]);
    kk = fmaf(k, k, kk);
  }
  const float unit = 1.f / sqrtf(warp_sum(kk) + kDeltaUnit);
  float rau = 0.f, rk = 0.f;
  for (int d = lane; d < DP; d += 32) {
    const bool in = d < D;
    const float k = in ? to_f(row[L.off_kk + o + d]) : 0.f, r = in ? to_f(row[L.off_r + o + d]) : 0.f, u = k * unit;
    const float x = in ? -kDecayScale * sigmoid_as<T>(to_f(low[o + d]) + L.w0[o + d]) : 0.f;
    const float au = in ? sigmoid_as<T>(to_f(row[L.off_a + o + d]) + L.a_b[o + d]) * u : 0.f;
    const float w = sizeof(T) == 2 ? __expf(x) : expf(x);
    s.u[d] = u;
    s.wr[d] = w * r;
    s.w[d] = sizeof(T) == 2 ? w : expm1f(x);
    s.k[d] = k;
    s.au[d] = au;
    s.v[d] = in ? to_f(row[L.off_vv + o + d]) : 0.f;
    rau = fmaf(r, au, rau);
    rk = fmaf(r, k, rk);
  }
  return make_float2(warp_sum(rau), warp_sum(rk));
}
// New value of a state element.
template <typename T>
__device__ __forceinline__ float delta_apply(float w, float s, float k, float v, float au, float us) {
  const float t = fmaf(k, v, -au * us);
  return sizeof(T) == 2 ? fmaf(w, s, t) : s + fmaf(w, s, t);
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
  const DeltaVecs s = DeltaVecs::at(vec, D);
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
      const float2 d = delta_token<T>(L, proj + (size_t)r * ld, low + (size_t)r * ldl, h, s, D);
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
      for (int i = kr; i < D; i += rows) S[i * D + j] = delta_apply<T>(s.w[i], S[i * D + j], s.k[i], v, s.au[i], us);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < D * D; i += DS_THREADS) state[i] = S[i];
}

// ---- state in registers.  A thread holds CT columns of DP / KL keys (the float4 groups q, q + KL, ... of lane
// q), so a token's vectors are read from shared memory without bank conflicts and two shuffles finish a dot
// product.  CW warps walk through the tokens; four others prepare the next DT_T tokens meanwhile.
constexpr int DT_T = 16, DT_PREP = 4;

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 x, y, z;\n\t"
      "mov.b64 x, {%2, %3};\n\tmov.b64 y, {%4, %5};\n\tmov.b64 z, {%6, %7};\n\t"
      "fma.rn.f32x2 z, x, y, z;\n\t"
      "mov.b64 {%0, %1}, z;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 x, y;\n\t"
      "mov.b64 x, {%2, %3};\n\tmov.b64 y, {%4, %5};\n\t"
      "mul.rn.f32x2 x, x, y;\n\t"
      "mov.b64 {%0, %1}, x;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

template <typename T, int DP, int CW>
__global__ void __launch_bounds__((CW + DT_PREP) * 32, 2)
hy_delta_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                     int ldl, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b) {
  constexpr int KT = 16, KL = DP / KT, CT = 2, PAIRS = KT / 2;
  constexpr int COLS = CW * (32 / KL) * CT;          // columns of a block
  constexpr int STRIDE = 6 * DP + 4;                 // floats of a token: vectors, then the two scalars
  extern __shared__ __align__(16) float sm[];        // [2][DT_T][STRIDE]
  const int seq = blockIdx.z, h = blockIdx.y, D = L.p;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = b.seq_row0[seq], n = b.seq_row0[seq + 1] - r0;
  auto prepare = [&](int t0, int w, int nw) {
    for (int t = w; t < DT_T && t0 + t < n; t += nw) {
      float* p = sm + (((t0 / DT_T) & 1) * DT_T + t) * STRIDE;
      const size_t r = r0 + t0 + t;
      const float2 d = delta_token<T>(L, proj + r * ld, low + r * ldl, h, DeltaVecs::at(p, DP), DP);
      if (lane == 0) *reinterpret_cast<float2*>(p + 6 * DP) = d;
    }
  };
  prepare(0, warp, CW + DT_PREP);
  __syncthreads();
  if (warp >= CW) {
    for (int t0 = 0; t0 < n; t0 += DT_T) {
      prepare(t0 + DT_T, warp - CW, DT_PREP);
      __syncthreads();
    }
    return;
  }
  const int q = lane % KL, c0 = blockIdx.x * COLS + (warp * (32 / KL) + lane / KL) * CT;
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.seq_pos0[seq] == 0;
  float2 S[CT][PAIRS];                               // two neighbouring keys of a column
  auto key = [&](int i) { return 4 * (q + KL * (i / 2)) + 2 * (i & 1); };
#pragma unroll
  for (int i = 0; i < PAIRS; ++i)
#pragma unroll
    for (int c = 0; c < CT; ++c) {
      const int k = key(i), col = c0 + c;
      S[c][i].x = !fresh && k < D && col < D ? state[(size_t)k * D + col] : 0.f;
      S[c][i].y = !fresh && k + 1 < D && col < D ? state[(size_t)(k + 1) * D + col] : 0.f;
    }
  T* yc = y + (size_t)r0 * ldy + h * L.pp + c0;
  const bool writes = q == 0 && c0 < L.pp;           // (pp is even: both columns or none)
  for (int t0 = 0; t0 < n; t0 += DT_T) {
    const int nt = min(DT_T, n - t0);
    const float* p = sm + ((t0 / DT_T) & 1) * DT_T * STRIDE;
    for (int t = 0; t < nt; ++t, p += STRIDE) {
      const float4* u4 = reinterpret_cast<const float4*>(p) + q;
      const float4* wr4 = u4 + DP / 4;
      float2 pu[CT], pr[CT];
#pragma unroll
      for (int c = 0; c < CT; ++c) pu[c] = pr[c] = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < PAIRS; i += 2) {
        const float4 u = u4[KL * (i / 2)], wr = wr4[KL * (i / 2)];
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          pu[c] = fma2(make_float2(u.x, u.y), S[c][i], pu[c]);
          pr[c] = fma2(make_float2(wr.x, wr.y), S[c][i], pr[c]);
          pu[c] = fma2(make_float2(u.z, u.w), S[c][i + 1], pu[c]);
          pr[c] = fma2(make_float2(wr.z, wr.w), S[c][i + 1], pr[c]);
        }
      }
      const float2 v = *reinterpret_cast<const float2*>(p + 5 * DP + min(c0, DP - CT));
      const float2 dots = *reinterpret_cast<const float2*>(p + 6 * DP);
      float us[CT], os[CT];
#pragma unroll
      for (int c = 0; c < CT; ++c) {
        us[c] = pu[c].x + pu[c].y;
        os[c] = pr[c].x + pr[c].y;
      }
#pragma unroll
      for (int o = 1; o < KL; o <<= 1)
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          us[c] += __shfl_xor_sync(0xffffffffu, us[c], o);
          os[c] += __shfl_xor_sync(0xffffffffu, os[c], o);
        }
      const float4* w4 = u4 + 2 * (DP / 4);
      const float4* k4 = u4 + 3 * (DP / 4);
      const float4* au4 = u4 + 4 * (DP / 4);
      const float vc[CT] = {v.x, v.y};
#pragma unroll
      for (int i = 0; i < PAIRS; i += 2) {
        const float4 w = w4[KL * (i / 2)], k = k4[KL * (i / 2)], au = au4[KL * (i / 2)];
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          const float2 vv = make_float2(vc[c], vc[c]), uu = make_float2(-us[c], -us[c]);
          S[c][i] = fma2(make_float2(w.x, w.y), S[c][i], fma2(make_float2(au.x, au.y), uu, mul2(make_float2(k.x, k.y), vv)));
          S[c][i + 1] =
              fma2(make_float2(w.z, w.w), S[c][i + 1], fma2(make_float2(au.z, au.w), uu, mul2(make_float2(k.z, k.w), vv)));
        }
      }
      if (writes) {
        struct alignas(sizeof(T) * 2) Two {
          T v[2];
        } o;
#pragma unroll
        for (int c = 0; c < CT; ++c) o.v[c] = from_f<T>(fmaf(dots.y, vc[c], fmaf(-dots.x, us[c], os[c])));
        *reinterpret_cast<Two*>(yc + (size_t)(t0 + t) * ldy) = o;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < PAIRS; ++i)
#pragma unroll
    for (int c = 0; c < CT; ++c) {
      const int k = key(i), col = c0 + c;
      if (k < D && col < D) state[(size_t)k * D + col] = S[c][i].x;
      if (k + 1 < D && col < D) state[(size_t)(k + 1) * D + col] = S[c][i].y;
    }
}

// ---- one token per sequence.  Lanes over four columns each, thread rows over keys, U keys of a thread.
template <typename T, int THREADS, int U>
__global__ void __launch_bounds__(THREADS)
hy_delta_decode_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ low,
                       int ldl, T* __restrict__ cat, int ldc, const __grid_constant__ BbHyBatch b, float eps) {
  extern __shared__ __align__(16) float sm[];
  const int seq = b.ns_pre + blockIdx.x, h = blockIdx.y, D = L.p, cv = D / 4;
  const size_t r = b.n_pre + blockIdx.x;
  int lanes = 1;
  while (lanes < cv) lanes <<= 1;
  const int lane = threadIdx.x % lanes, kr = threadIdx.x / lanes, rows = THREADS / lanes;
  const DeltaVecs s = DeltaVecs::at(sm, D);
  float* red = sm + 6 * D;                           // [rows][2][D]
  float* out = red + rows * 2 * D;                   // [D]
  __shared__ float dots[2];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * D * D;
  const bool fresh = b.pos[r] == 0, mine = lane < cv;
  float4 S[U];
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const int k = kr + i * rows;
    S[i] = !fresh && mine && k < D ? reinterpret_cast<const float4*>(state + (size_t)k * D)[lane] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (threadIdx.x < 32) {
    const float2 d = delta_token<T>(L, proj + r * ld, low + r * ldl, h, s, D);
    if (threadIdx.x == 0) {
      dots[0] = d.x;
      dots[1] = d.y;
    }
  }
  __syncthreads();
  float4 pu = make_float4(0.f, 0.f, 0.f, 0.f), pr = pu;
#pragma unroll
  for (int i = 0; i < U; ++i) {
    const int k = kr + i * rows;
    if (k < D) {
      const float u = s.u[k], w = s.wr[k];
      pu.x = fmaf(u, S[i].x, pu.x); pu.y = fmaf(u, S[i].y, pu.y); pu.z = fmaf(u, S[i].z, pu.z); pu.w = fmaf(u, S[i].w, pu.w);
      pr.x = fmaf(w, S[i].x, pr.x); pr.y = fmaf(w, S[i].y, pr.y); pr.z = fmaf(w, S[i].z, pr.z); pr.w = fmaf(w, S[i].w, pr.w);
    }
  }
  if (mine) {
    reinterpret_cast<float4*>(red + (kr * 2) * D)[lane] = pu;
    reinterpret_cast<float4*>(red + (kr * 2 + 1) * D)[lane] = pr;
  }
  __syncthreads();
  if (mine) {
    float4 us = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int q = 0; q < rows; ++q) {
      const float4 a = reinterpret_cast<const float4*>(red + (q * 2) * D)[lane];
      us.x += a.x; us.y += a.y; us.z += a.z; us.w += a.w;
    }
    const float4 v = reinterpret_cast<const float4*>(s.v)[lane];
    if (kr == 0) {
      float4 os = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int q = 0; q < rows; ++q) {
        const float4 a = reinterpret_cast<const float4*>(red + (q * 2 + 1) * D)[lane];
        os.x += a.x; os.y += a.y; os.z += a.z; os.w += a.w;
      }
      // the same rounding of the recurrence's output as in a prompt portion
      auto fin = [&](float o, float u, float x) { return to_f(from_f<T>(fmaf(dots[1], x, fmaf(-dots[0], u, o)))); };
      reinterpret_cast<float4*>(out)[lane] =
          make_float4(fin(os.x, us.x, v.x), fin(os.y, us.y, v.y), fin(os.z, us.z, v.z), fin(os.w, us.w, v.w));
    }
#pragma unroll
    for (int i = 0; i < U; ++i) {
      const int k = kr + i * rows;
      if (k < D) {
        const float w = s.w[k], kk = s.k[k], au = s.au[k];
        reinterpret_cast<float4*>(state + (size_t)k * D)[lane] =
            make_float4(delta_apply<T>(w, S[i].x, kk, v.x, au, us.x), delta_apply<T>(w, S[i].y, kk, v.y, au, us.y),
                        delta_apply<T>(w, S[i].z, kk, v.z, au, us.z), delta_apply<T>(w, S[i].w, kk, v.w, au, us.w));
      }
    }
  }
  __syncthreads();
  if (threadIdx.x < 32) {
    const int o = h * L.pp;
    float ss = 0.f;
    for (int d = threadIdx.x; d < D; d += 32) ss = fmaf(out[d], out[d], ss);
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
    for (int d = threadIdx.x; d < L.pp; d += 32)
      cat[r * ldc + o + d] = from_f<T>(
          d < D ? out[d] * rstd * L.gnorm[o + d] * sigmoid_as<T>(to_f(proj[r * ld + L.off_gg + o + d])) : 0.f);
  }
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
static int launch_scan_any(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int seq0, int n_seq, cudaStream_t s) {
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

template <int DP, int CW>
static int launch_scan_regs(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  using T = __nv_bfloat16;
  static PerDeviceOnce once;
  constexpr int smem = 2 * DT_T * (6 * DP + 4) * 4, cols = CW * (32 / (DP / 16)) * 2;
  const cudaError_t e = ensure_dyn_smem(once, hy_delta_scan_kernel<T, DP, CW>, smem);
  if (e != cudaSuccess) return (int)e;
  hy_delta_scan_kernel<T, DP, CW><<<dim3((L.p + cols - 1) / cols, L.heads, b.ns_pre), (CW + DT_PREP) * 32, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.y), w.ld_y, b);
  return (int)cudaGetLastError();
}

// Few heads: the columns of a head are spread over more blocks.
static int launch_scan_bf16(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  const long pairs = (long)b.ns_pre * L.heads;
  const int sms = sm_count();
  if (L.p <= 32) return launch_scan_regs<32, 1>(L, w, b, s);
  if (L.p <= 64) {
    if (pairs * 4 <= sms) return launch_scan_regs<64, 1>(L, w, b, s);
    return pairs <= sms ? launch_scan_regs<64, 2>(L, w, b, s) : launch_scan_regs<64, 4>(L, w, b, s);
  }
  if (L.p <= 128) return pairs * 8 <= sms ? launch_scan_regs<128, 2>(L, w, b, s) : launch_scan_regs<128, 4>(L, w, b, s);
  return BB_ESIZE;
}

template <typename T, int THREADS, int U>
static int launch_decode_u(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  int lanes = 1;
  while (lanes < L.p / 4) lanes <<= 1;
  const size_t smem = 4ull * (7 + 2 * (THREADS / lanes)) * L.p;
  if (smem > 48 * 1024) return BB_ESIZE;
  hy_delta_decode_kernel<T, THREADS, U><<<dim3(b.ns - b.ns_pre, L.heads), THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.aux), w.ld_aux, static_cast<T*>(w.cat), w.ld_cat, b, eps);
  return (int)cudaGetLastError();
}
template <typename T>
static int launch_decode(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  if (L.p % 4 || L.p > 128) return BB_ESIZE;
  if (L.p <= 32) return launch_decode_u<T, 128, 2>(L, w, b, eps, s);
  if (L.p <= 64) return launch_decode_u<T, 128, 8>(L, w, b, eps, s);
  return launch_decode_u<T, 256, 16>(L, w, b, eps, s);
}

template <typename T>
static int launch_post(const BbHyLayer& L, const BbHyWork& w, int rows, float eps, cudaStream_t s) {
  const int grid = (int)(((long)rows * L.heads * 32 + 127) / 128);
  hy_delta_post_kernel<T><<<grid, 128, 0, s>>>(L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.y), w.ld_y,
                                               static_cast<T*>(w.cat), w.ld_cat, rows, eps);
  return (int)cudaGetLastError();
}

template <typename T>
static int run_delta(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  const int n_dec = b.ns - b.ns_pre;
  int post = b.n_pre;                    // rows whose outputs are still to be normed and gated
  if (n_dec > 0) {
    int rc = launch_decode<T>(L, w, b, eps, s);
    if (rc == BB_ESIZE) {
      rc = launch_scan_any<T>(L, w, b, b.ns_pre, n_dec, s);
      post = b.n;
    }
    if (rc) return rc;
  }
  if (b.ns_pre > 0) {
    int rc = sizeof(T) == 2 ? launch_scan_bf16(L, w, b, s) : BB_ESIZE;
    if (rc == BB_ESIZE) rc = launch_scan_any<T>(L, w, b, 0, b.ns_pre, s);
    if (rc) return rc;
  }
  return post > 0 ? launch_post<T>(L, w, post, eps, s) : BB_OK;
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

// Recurrence, norm and gate of every row of the step -> w->cat.
BB_API int bb_hy_delta(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? run_delta<float>(*L, *w, *b, c->eps, (cudaStream_t)stream)
                  : run_delta<__nv_bfloat16>(*L, *w, *b, c->eps, (cudaStream_t)stream);
}

// The recurrence of the prompt portions alone -> w->y; `any`: by the kernel that covers every size.
BB_API int bb_hy_delta_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int any, void* stream) {
  cudaStream_t s = (cudaStream_t)stream;
  if (b->ns_pre <= 0) return BB_OK;
  if (c->dtype) return launch_scan_any<float>(*L, *w, *b, 0, b->ns_pre, s);
  return any ? launch_scan_any<__nv_bfloat16>(*L, *w, *b, 0, b->ns_pre, s) : launch_scan_bf16(*L, *w, *b, s);
}

// Mamba-2 mixer kernels (fp32 state and recurrence; bf16 or fp32 projections and convolution).
//   hy_conv         causal per-channel convolution + bias (+ silu) over packed rows; taps that reach back
//                   before a portion come from the sequence's state slot.  The same launch turns raw step
//                   sizes, where a layer has them, into softplus(dt + bias).  Inputs may carry a bias of their
//                   own, which places before the start of the sequence do not have.
//   hy_ssm_scan     recurrence of a prompt portion, one token after the other, one block per (sequence,
//                   head): any sizes, fp32 throughout
//   hy_ssm_decode   one token per sequence: convolution, step size, state update and output in one
//                   kernel, one block per (sequence, head); the state is read and written once
// State layout: ssm [slot][head][n][p] fp32; convolution ring [slot][taps - 1][channels], the raw input of
// position p at p % (taps - 1).  A sequence at position 0 starts from zeros whatever its slot holds, so
// slots need no clearing.
#include "../common/host.hpp"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int CONV_ROWS = 8;   // consecutive rows of a thread in portions, their inputs asked for together

template <typename T>
struct alignas(sizeof(T) * 4) Raw4 {
  T v[4];
};

// Raw convolution input of row r, k tokens back, 4 channels from c: from the portion itself, from the
// sequence's slot, or zeros before its start.
template <typename T>
__device__ __forceinline__ Raw4<T> conv_tap(const BbHyLayer& L, const T* proj, int ld, int r, int k, int c, int pos,
                                            int pos0, int slot) {
  if (k <= pos - pos0) return *reinterpret_cast<const Raw4<T>*>(proj + (size_t)(r - k) * ld + L.off_xbc + c);
  if (k <= pos) {
    const int keep = L.taps - 1;
    return *reinterpret_cast<const Raw4<T>*>(static_cast<const T*>(L.conv_state) +
                                             ((size_t)slot * keep + (pos - k) % keep) * L.chp + c);
  }
  Raw4<T> z;
#pragma unroll
  for (int j = 0; j < 4; ++j) z.v[j] = from_f<T>(0.f);
  return z;
}

// TAPS = 4 keeps a thread's inputs in registers as they are stored; TAPS = 0 reads every tap again (any
// length).
template <typename T, int TAPS, bool SILU, int ROWS>
__global__ void __launch_bounds__(128, sizeof(T) == 2 ? 7 : 5)
hy_conv_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, T* __restrict__ xbc, int ldx,
               float* __restrict__ dt, int lddt, const __grid_constant__ BbHyBatch b, int row0, int rows) {
  const int cv = blockIdx.x * 128 + threadIdx.x;   // vector of 4 channels, then vectors of 4 step sizes
  const int nch = L.chp / 4, ndt = (L.heads + 7) / 8 * 2;
  const int r0 = row0 + blockIdx.y * ROWS, r1 = min(r0 + ROWS, row0 + rows);
  if (cv >= nch + ndt) return;
  if (cv >= nch) {
    const int h0 = (cv - nch) * 4;
    const float4 bias = *reinterpret_cast<const float4*>(L.dt_bias + h0);
#pragma unroll 4
    for (int r = r0; r < r1; ++r) {
      const Raw4<T> f = *reinterpret_cast<const Raw4<T>*>(proj + (size_t)r * ld + L.off_dt + h0);
      *reinterpret_cast<float4*>(dt + (size_t)r * lddt + h0) =
          make_float4(softplus_f(to_f(f.v[0]) + bias.x), softplus_f(to_f(f.v[1]) + bias.y),
                      softplus_f(to_f(f.v[2]) + bias.z), softplus_f(to_f(f.v[3]) + bias.w));
    }
    return;
  }
  const int c = cv * 4;
  const float4 bias4 = *reinterpret_cast<const float4*>(L.conv_b + c);
  const float bias[4] = {bias4.x, bias4.y, bias4.z, bias4.w};
  float xb[4] = {0.f, 0.f, 0.f, 0.f};              // bias of the inputs
  if (!SILU) {
    const float4 t = *reinterpret_cast<const float4*>(L.x_b + c);
    xb[0] = t.x; xb[1] = t.y; xb[2] = t.z; xb[3] = t.w;
  }
  if constexpr (TAPS > 0) {
    constexpr int K = TAPS - 1;
    Raw4<T> raw[ROWS + K];   // raw[K + i]: row r0 + i; before it the inputs ahead of r0
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
      if (r0 + i < r1) raw[K + i] = *reinterpret_cast<const Raw4<T>*>(proj + (size_t)(r0 + i) * ld + L.off_xbc + c);
    // the rows before r0 are asked for before it is known whether they are this sequence's
#pragma unroll
    for (int k = 1; k <= K; ++k)
      if (ROWS > 1 && r0 >= k) raw[K - k] = *reinterpret_cast<const Raw4<T>*>(proj + (size_t)(r0 - k) * ld + L.off_xbc + c);
    int last_seq = b.row_seq[r0];
    const bool one = last_seq == b.row_seq[r1 - 1];   // all rows of this thread belong to one sequence
    {
      const int pos = b.pos[r0], pos0 = b.seq_pos0[last_seq], slot = b.seq_slot[last_seq];
#pragma unroll
      for (int k = 1; k <= K; ++k)
        if (k > pos - pos0) raw[K - k] = conv_tap(L, proj, ld, r0, k, c, pos, pos0, slot);
    }
    float w[TAPS][4];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      const float4 t = *reinterpret_cast<const float4*>(L.conv_w + (size_t)k * L.chp + c);
      w[k][0] = t.x; w[k][1] = t.y; w[k][2] = t.z; w[k][3] = t.w;
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = r0 + i;
      if (r >= r1) break;
      if (!one) {
        const int seq = b.row_seq[r];
        if (seq != last_seq) {    // a sequence starts inside: what lies ahead of it is its own
          const int pos = b.pos[r], pos0 = b.seq_pos0[seq], slot = b.seq_slot[seq];
#pragma unroll
          for (int k = 1; k <= K; ++k) raw[K + i - k] = conv_tap(L, proj, ld, r, k, c, pos, pos0, slot);
          last_seq = seq;
        }
      }
      Raw4<T> o;
      const int first = SILU ? 0 : K - b.pos[r];       // taps before it lie ahead of the sequence
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float s = bias[j];
#pragma unroll
        for (int k = 0; k < TAPS; ++k)
          s = fmaf(w[k][j], SILU ? to_f(raw[i + k].v[j]) : (k >= first ? to_f(raw[i + k].v[j]) + xb[j] : 0.f), s);
        o.v[j] = from_f<T>(SILU ? silu_as<T>(s) : s);
      }
      *reinterpret_cast<Raw4<T>*>(xbc + (size_t)r * ldx + c) = o;
    }
  } else {
    for (int r = r0; r < r1; ++r) {
      const int seq = b.row_seq[r];
      const int pos = b.pos[r], pos0 = b.seq_pos0[seq], slot = b.seq_slot[seq];
      float s[4] = {bias[0], bias[1], bias[2], bias[3]};
      for (int k = L.taps - 1; k >= 0; --k) {
        const Raw4<T> u = conv_tap(L, proj, ld, r, k, c, pos, pos0, slot);
        const float* w = L.conv_w + (size_t)(L.taps - 1 - k) * L.chp + c;
#pragma unroll
        for (int j = 0; j < 4; ++j) s[j] = fmaf(w[j], k <= pos ? to_f(u.v[j]) + xb[j] : 0.f, s[j]);
      }
      Raw4<T> o;
#pragma unroll
      for (int j = 0; j < 4; ++j) o.v[j] = from_f<T>(SILU ? silu_as<T>(s[j]) : s[j]);
      *reinterpret_cast<Raw4<T>*>(xbc + (size_t)r * ldx + c) = o;
    }
  }
}

// Lanes over p (a power of two of them), thread rows over n.
struct SsmMap {
  int lanes, rows, lane, row;
};
__device__ __forceinline__ SsmMap ssm_map(int p, int threads) {
  int lanes = 1;
  while (lanes < p && lanes < 32) lanes <<= 1;
  return {lanes, threads / lanes, (int)threadIdx.x % lanes, (int)threadIdx.x / lanes};
}

constexpr int SCAN_T = 8;   // tokens staged at a time
constexpr int SCAN_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(SCAN_THREADS)
hy_ssm_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ xbc, int ldx, const float* __restrict__ dt,
                   int lddt, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b) {
  extern __shared__ float sm[];
  const int seq = blockIdx.x, h = blockIdx.y, g = h / (L.heads / L.groups);
  const int N = L.n, P = L.p;
  const SsmMap m = ssm_map(P, SCAN_THREADS);
  float* S = sm;                        // [N][P]
  float* sx = S + N * P;                // [SCAN_T][P]
  float* sB = sx + SCAN_T * P;          // [SCAN_T][N]
  float* sC = sB + SCAN_T * N;
  float* red = sC + SCAN_T * N;         // [rows][P]
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1], slot = b.seq_slot[seq];
  float* state = L.ssm_state + ((size_t)slot * L.heads + h) * N * P;
  const bool fresh = b.seq_pos0[seq] == 0;
  for (int i = threadIdx.x; i < N * P; i += SCAN_THREADS) S[i] = fresh ? 0.f : state[i];
  const float a = L.a[h], D = L.d_skip[h];
  for (int t0 = r0; t0 < r1; t0 += SCAN_T) {
    const int nt = min(SCAN_T, r1 - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * P; i += SCAN_THREADS)
      sx[i] = to_f(xbc[(size_t)(t0 + i / P) * ldx + h * P + i % P]);
    for (int i = threadIdx.x; i < nt * N; i += SCAN_THREADS) {
      const T* row = xbc + (size_t)(t0 + i / N) * ldx + L.inner + g * N + i % N;
      sB[i] = to_f(row[0]);
      sC[i] = to_f(row[(size_t)L.groups * N]);
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float d = dt[(size_t)(t0 + t) * lddt + h];
      const float decay = expf(a * d);
      for (int p = m.lane; p < P; p += m.lanes) {
        const float dx = d * sx[t * P + p];
        float acc = 0.f;
        for (int n = m.row; n < N; n += m.rows) {
          const float s = fmaf(decay, S[n * P + p], sB[t * N + n] * dx);
          S[n * P + p] = s;
          acc = fmaf(sC[t * N + n], s, acc);
        }
        red[m.row * P + p] = acc;
      }
      __syncthreads();
      for (int p = threadIdx.x; p < P; p += SCAN_THREADS) {
        float acc = 0.f;
        for (int q = 0; q < m.rows; ++q) acc += red[q * P + p];
        y[(size_t)(t0 + t) * ldy + h * P + p] = from_f<T>(acc + D * sx[t * P + p]);
      }
      __syncthreads();
    }
  }
  for (int i = threadIdx.x; i < N * P; i += SCAN_THREADS) state[i] = S[i];
}

constexpr int DEC_THREADS = 128;

// V: state elements of a lane (4: 16-byte accesses, p % 4 == 0; 1: any p).
template <typename T, int V>
__global__ void __launch_bounds__(DEC_THREADS)
hy_ssm_decode_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, T* __restrict__ y, int ldy,
                     const __grid_constant__ BbHyBatch b) {
  extern __shared__ float sm[];
  const int seq = b.ns_pre + blockIdx.x, r = b.n_pre + blockIdx.x, h = blockIdx.y;
  const int N = L.n, P = L.p, g = h / (L.heads / L.groups);
  float* sx = sm;              // [P]
  float* sB = sx + P;          // [N]
  float* sC = sB + N;          // [N]
  float* red = sm + ((P + 2 * N + 3) & ~3);   // [rows][P]
  const int pos = b.pos[r], slot = b.seq_slot[seq];
  const T* row = proj + (size_t)r * ld;
  float* state = L.ssm_state + ((size_t)slot * L.heads + h) * N * P;
  const int pv = P / V;
  int lanes = 1;
  while (lanes < pv && lanes < 32) lanes <<= 1;
  const int lane = threadIdx.x % lanes, nr = threadIdx.x / lanes, rows = DEC_THREADS / lanes;
  constexpr int U = 8;         // state vectors in flight: the first batch is asked for before anything else
  float s[U][V];
  auto fetch = [&](int n0, int p) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int n = n0 + u * rows;
      if (n < N && p < pv) {
        if constexpr (V == 4) {
          const float4 v = reinterpret_cast<const float4*>(state + (size_t)n * P)[p];
          s[u][0] = v.x; s[u][1] = v.y; s[u][2] = v.z; s[u][3] = v.w;
        } else {
          s[u][0] = state[(size_t)n * P + p];
        }
      }
    }
  };
  const bool fresh = pos == 0;
  fetch(nr, lane);
  const float d = softplus_f(to_f(row[L.off_dt + h]) + L.dt_bias[h]);
  const float decay = fresh ? 0.f : expf(L.a[h] * d);
  const int keep = L.taps - 1;
  const T* ring = static_cast<const T*>(L.conv_state) + (size_t)slot * keep * L.chp;
  for (int i = threadIdx.x; i < P + 2 * N; i += DEC_THREADS) {
    const int c = i < P ? h * P + i : (i < P + N ? L.inner + g * N + (i - P) : L.inner + (L.groups + g) * N + (i - P - N));
    float acc = L.conv_b[c];
    for (int k = min(keep, pos); k > 0; --k)
      acc = fmaf(L.conv_w[(size_t)(keep - k) * L.chp + c], to_f(ring[(size_t)((pos - k) % keep) * L.chp + c]), acc);
    acc = fmaf(L.conv_w[(size_t)keep * L.chp + c], to_f(row[L.off_xbc + c]), acc);
    // the same rounding of the convolution's output as in a prompt portion
    sm[i] = to_f(from_f<T>(silu_as<T>(acc)));
  }
  __syncthreads();
  for (int p = lane; p < pv; p += lanes) {
    float dx[V], acc[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      dx[j] = d * sx[p * V + j];
      acc[j] = 0.f;
    }
    for (int n0 = nr; n0 < N; n0 += U * rows) {
      if (p != lane || n0 != nr) fetch(n0, p);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * rows;
        if (n < N) {
          const float bn = sB[n], cn = sC[n];
#pragma unroll
          for (int j = 0; j < V; ++j) {
            // a fresh sequence ignores whatever its slot holds (0 * stale could be NaN)
            s[u][j] = fresh ? bn * dx[j] : fmaf(decay, s[u][j], bn * dx[j]);
            acc[j] = fmaf(cn, s[u][j], acc[j]);
          }
          if constexpr (V == 4)
            reinterpret_cast<float4*>(state + (size_t)n * P)[p] = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
          else
            state[(size_t)n * P + p] = s[u][0];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) red[nr * P + p * V + j] = acc[j];
  }
  __syncthreads();
  for (int p = threadIdx.x; p < P; p += DEC_THREADS) {
    float acc = 0.f;
    for (int q = 0; q < rows; ++q) acc += red[q * P + p];
    y[(size_t)r * ldy + h * P + p] = from_f<T>(acc + L.d_skip[h] * sx[p]);
  }
}

template <typename T, bool SILU, int ROWS>
static int launch_conv(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int row0, int rows, cudaStream_t s) {
  const int vecs = L.chp / 4 + (L.heads + 7) / 8 * 2;
  dim3 grid((vecs + 127) / 128, (rows + ROWS - 1) / ROWS);
  if (grid.y > 65535) return BB_ESIZE;
  const T* proj = static_cast<const T*>(w.proj);
  T* xbc = static_cast<T*>(w.xbc);
  if (L.taps == 4) hy_conv_kernel<T, 4, SILU, ROWS><<<grid, 128, 0, s>>>(L, proj, w.ld_proj, xbc, w.ld_xbc, w.dt, w.ld_dt, b, row0, rows);
  else hy_conv_kernel<T, 0, SILU, ROWS><<<grid, 128, 0, s>>>(L, proj, w.ld_proj, xbc, w.ld_xbc, w.dt, w.ld_dt, b, row0, rows);
  return (int)cudaGetLastError();
}

static int lanes_of(int p) {
  int l = 1;
  while (l < p && l < 32) l <<= 1;
  return l;
}

template <typename T>
static int launch_scan(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once;
  const int rows = SCAN_THREADS / lanes_of(L.p);
  const size_t smem = 4ull * ((size_t)L.n * L.p + SCAN_T * (L.p + 2 * L.n) + (size_t)rows * L.p);
  if (smem > 220 * 1024) return BB_ESIZE;
  if (smem > 40 * 1024) {
    const cudaError_t e = ensure_dyn_smem(once, hy_ssm_scan_kernel<T>, 220 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  hy_ssm_scan_kernel<T><<<dim3(b.ns_pre, L.heads), SCAN_THREADS, smem, s>>>(
      L, static_cast<const T*>(w.xbc), w.ld_xbc, w.dt, w.ld_dt, static_cast<T*>(w.y), w.ld_y, b);
  return (int)cudaGetLastError();
}

template <typename T, int V>
static int launch_decode_v(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once;
  const int rows = DEC_THREADS / lanes_of(L.p / V);
  const size_t smem = 4ull * (((L.p + 2 * L.n + 3) & ~3) + (size_t)rows * L.p);
  if (smem > 200 * 1024) return BB_ESIZE;
  if (smem > 40 * 1024) {
    const cudaError_t e = ensure_dyn_smem(once, hy_ssm_decode_kernel<T, V>, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  hy_ssm_decode_kernel<T, V><<<dim3(b.ns - b.ns_pre, L.heads), DEC_THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<T*>(w.y), w.ld_y, b);
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

BB_API int bb_hy_conv(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->n_pre <= 0) return BB_OK;
  return c->dtype ? launch_conv<float, true, CONV_ROWS>(*L, *w, *b, 0, b->n_pre, (cudaStream_t)stream)
                  : launch_conv<__nv_bfloat16, true, CONV_ROWS>(*L, *w, *b, 0, b->n_pre, (cudaStream_t)stream);
}

// The same without activation, with the inputs' bias x_b, for every row of the step.
BB_API int bb_hy_conv_linear(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  cudaStream_t s = (cudaStream_t)stream;
  const int dec = b->n - b->n_pre;       // rows of different sequences: one to a thread
  int rc = BB_OK;
  if (b->n_pre > 0)
    rc = c->dtype ? launch_conv<float, false, CONV_ROWS>(*L, *w, *b, 0, b->n_pre, s)
                  : launch_conv<__nv_bfloat16, false, CONV_ROWS>(*L, *w, *b, 0, b->n_pre, s);
  if (rc == BB_OK && dec > 0)
    rc = c->dtype ? launch_conv<float, false, 1>(*L, *w, *b, b->n_pre, dec, s)
                  : launch_conv<__nv_bfloat16, false, 1>(*L, *w, *b, b->n_pre, dec, s);
  return rc;
}

BB_API int bb_hy_ssm_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->ns_pre <= 0) return BB_OK;
  return c->dtype ? launch_scan<float>(*L, *w, *b, (cudaStream_t)stream)
                  : launch_scan<__nv_bfloat16>(*L, *w, *b, (cudaStream_t)stream);
}

BB_API int bb_hy_ssm_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->ns <= b->ns_pre) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  if (L->p % 4 == 0)
    return c->dtype ? launch_decode_v<float, 4>(*L, *w, *b, s) : launch_decode_v<__nv_bfloat16, 4>(*L, *w, *b, s);
  return c->dtype ? launch_decode_v<float, 1>(*L, *w, *b, s) : launch_decode_v<__nv_bfloat16, 1>(*L, *w, *b, s);
}

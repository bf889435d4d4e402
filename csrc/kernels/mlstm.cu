// Matrix memory with exponential gates (mLSTM; fp32 state and recurrence, bf16 or fp32 projections).  Per head,
// with log gates i = cap tanh((. + bias) / cap) and f = logsigmoid(cap tanh((. + bias) / cap)) of fp32 products:
//   m' = max(f + m, i),  keep = exp(f + m - m'),  add = exp(i - m')
//   S <- keep S + add k v^T,   n <- keep n + add k,   o = S^T q / (max(|n.q|, exp(-m')) + 1e-6)
// and the head's output is o over its root mean square, times a gain and a sigmoid gate.
//   hy_mlstm_gates    log gates of the prompt portions, in place, for the chunked kernel
//   hy_mlstm_scan     prompt portions one token after the other, one block per (sequence, head, value columns):
//                     any sizes, fp32 throughout
//   hy_mlstm_decode   one token per sequence: gates, state, norm and output gate in one kernel; the state is read
//                     and written once
// State of a head: S [n][p], normaliser [n], m.  A sequence at position 0 starts from zeros (m too) whatever its
// slot holds.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr float kMemoryEps = 1e-6f;

struct LogGates {
  float i, f;
};
__device__ __forceinline__ LogGates log_gates(const BbHyLayer& L, float raw_i, float raw_f, int h) {
  const float x = L.gate_cap * tanhf((raw_f + L.f_b[h]) / L.gate_cap);
  return {L.gate_cap * tanhf((raw_i + L.i_b[h]) / L.gate_cap), fminf(x, 0.f) - log1pf(expf(-fabsf(x)))};
}

__global__ void __launch_bounds__(128)
hy_mlstm_gates_kernel(const __grid_constant__ BbHyLayer L, float* __restrict__ g, int ld, int rows) {
  const int t = blockIdx.x * 128 + threadIdx.x, r = t / L.heads, h = t - r * L.heads;
  if (r >= rows) return;
  float *pi = g + (size_t)r * ld + L.off32_i + h, *pf = g + (size_t)r * ld + L.off32_f + h;
  const LogGates x = log_gates(L, *pi, *pf, h);
  *pi = x.i;
  *pf = x.f;
}

constexpr int MS_THREADS = 256, MS_T = 8;   // tokens staged at a time

// Value columns [c0, c0 + pc) of every head; `last`: the launch that writes the normaliser and the maximum (those
// before it read what it overwrites).
template <typename T>
__global__ void __launch_bounds__(MS_THREADS)
hy_mlstm_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const float* __restrict__ raw,
                     int ldr, T* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b, int seq0, int c0, int pc, int last) {
  extern __shared__ float sm[];
  const int seq = seq0 + blockIdx.x, h = blockIdx.y, N = L.n, P = min(pc, L.p - c0);
  int lanes = 1;
  while (lanes < pc && lanes < 32) lanes <<= 1;
  const int lane = threadIdx.x % lanes, nr = threadIdx.x / lanes, rows = MS_THREADS / lanes;
  float* S = sm;                        // [N][pc]
  float* nn = S + N * pc;               // [N]
  float* sq = nn + N;                   // [MS_T][N]
  float* sk = sq + MS_T * N;
  float* sv = sk + MS_T * N;            // [MS_T][pc]
  float* red = sv + MS_T * pc;          // [rows][pc]
  __shared__ float si[MS_T], sf[MS_T], s_nq;
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * L.mem;
  const bool fresh = b.seq_pos0[seq] == 0;
  for (int i = threadIdx.x; i < N * pc; i += MS_THREADS)
    S[i] = fresh || i % pc >= P ? 0.f : state[(size_t)(i / pc) * L.p + c0 + i % pc];
  for (int i = threadIdx.x; i < N; i += MS_THREADS) nn[i] = fresh ? 0.f : state[(size_t)N * L.p + i];
  float m = fresh ? 0.f : state[(size_t)N * L.p + N];
  for (int t0 = r0; t0 < r1; t0 += MS_T) {
    const int nt = min(MS_T, r1 - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * N; i += MS_THREADS) {
      const T* row = proj + (size_t)(t0 + i / N) * ld + h * L.np + i % N;
      sq[i] = to_f(row[L.off_q]) * L.q_scale;
      sk[i] = to_f(row[L.off_kk]);
    }
    for (int i = threadIdx.x; i < nt * pc; i += MS_THREADS)
      sv[i] = i % pc < P ? to_f(proj[(size_t)(t0 + i / pc) * ld + L.off_vv + h * L.pp + c0 + i % pc]) : 0.f;
    if (threadIdx.x < nt) {
      const float* g = raw + (size_t)(t0 + threadIdx.x) * ldr + h;
      const LogGates x = log_gates(L, g[L.off32_i], g[L.off32_f], h);
      si[threadIdx.x] = x.i;
      sf[threadIdx.x] = x.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float mn = fmaxf(sf[t] + m, si[t]), keep = expf(sf[t] + m - mn), add = expf(si[t] - mn);
      m = mn;
      const float *q = sq + t * N, *k = sk + t * N, *v = sv + t * pc;
      if (threadIdx.x < 32) {
        float a = 0.f;
        for (int d = threadIdx.x; d < N; d += 32) {
          const float x = fmaf(keep, nn[d], add * k[d]);
          nn[d] = x;
          a = fmaf(x, q[d], a);
        }
        a = warp_sum(a);
        if (threadIdx.x == 0) s_nq = a;
      }
      for (int p = lane; p < pc; p += lanes) {
        const float av = add * v[p];
        float acc = 0.f;
        for (int d = nr; d < N; d += rows) {
          const float s = fmaf(keep, S[d * pc + p], k[d] * av);
          S[d * pc + p] = s;
          acc = fmaf(q[d], s, acc);
        }
        red[nr * pc + p] = acc;
      }
      __syncthreads();
      const float den = fmaxf(fabsf(s_nq), expf(-m)) + kMemoryEps;
      for (int p = threadIdx.x; p < P; p += MS_THREADS) {
        float acc = 0.f;
        for (int x = 0; x < rows; ++x) acc += red[x * pc + p];
        y[(size_t)(t0 + t) * ldy + h * L.pp + c0 + p] = from_f<T>(acc / den);
      }
      __syncthreads();
    }
  }
  for (int i = threadIdx.x; i < N * pc; i += MS_THREADS)
    if (i % pc < P) state[(size_t)(i / pc) * L.p + c0 + i % pc] = S[i];
  if (last) {
    for (int i = threadIdx.x; i < N; i += MS_THREADS) state[(size_t)N * L.p + i] = nn[i];
    if (threadIdx.x == 0) state[(size_t)N * L.p + N] = m;
  }
}

// V: state elements of a lane (4: 16-byte accesses, p % 4 == 0; 1: any p).
template <typename T, int V, int THREADS>
__global__ void __launch_bounds__(THREADS)
hy_mlstm_decode_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const float* __restrict__ raw,
                       int ldr, T* __restrict__ cat, int ldc, const __grid_constant__ BbHyBatch b, float eps) {
  extern __shared__ float sm[];
  const int seq = b.ns_pre + blockIdx.x, h = blockIdx.y, N = L.n, P = L.p;
  const size_t r = b.n_pre + blockIdx.x;
  float* sv = sm;              // [P], then the outputs
  float* sq = sv + P;          // [N]
  float* sk = sq + N;          // [N]
  float* red = sm + ((P + 2 * N + 3) & ~3);   // [rows][P]
  __shared__ float part[2][32];
  const T* row = proj + r * ld;
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * L.mem;
  float* norm = state + (size_t)N * P;
  const int pv = P / V;
  int lanes = 1;
  while (lanes < pv && lanes < 32) lanes <<= 1;
  const int lane = threadIdx.x % lanes, nr = threadIdx.x / lanes, rows = THREADS / lanes;
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
  const bool fresh = b.pos[r] == 0;
  fetch(nr, lane);
  __shared__ float s_gate[3];
  if (threadIdx.x == 0) {
    const LogGates g = log_gates(L, raw[r * ldr + L.off32_i + h], raw[r * ldr + L.off32_f + h], h);
    const float m0 = fresh ? 0.f : norm[N], m = fmaxf(g.f + m0, g.i);
    s_gate[0] = m;
    s_gate[1] = expf(g.i - m);
    s_gate[2] = fresh ? 0.f : expf(g.f + m0 - m);
    norm[N] = m;
  }
  for (int p = threadIdx.x; p < P; p += THREADS) sv[p] = to_f(row[L.off_vv + h * L.pp + p]);
  __syncthreads();
  const float m = s_gate[0], add = s_gate[1], keep = s_gate[2];
  float nq = 0.f;
  for (int d = threadIdx.x; d < N; d += THREADS) {
    const float q = to_f(row[L.off_q + h * L.np + d]) * L.q_scale, k = to_f(row[L.off_kk + h * L.np + d]);
    sq[d] = q;
    sk[d] = k;
    // a fresh sequence ignores whatever its slot holds (0 * stale could be NaN)
    const float x = fresh ? add * k : fmaf(keep, norm[d], add * k);
    norm[d] = x;
    nq = fmaf(x, q, nq);
  }
  nq = block_sum(nq, part[0]);       // (its barrier also orders shared memory)
  for (int p = lane; p < pv; p += lanes) {
    float av[V], acc[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      av[j] = add * sv[p * V + j];
      acc[j] = 0.f;
    }
    for (int n0 = nr; n0 < N; n0 += U * rows) {
      if (p != lane || n0 != nr) fetch(n0, p);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * rows;
        if (n < N) {
          const float k = sk[n], q = sq[n];
#pragma unroll
          for (int j = 0; j < V; ++j) {
            s[u][j] = fresh ? k * av[j] : fmaf(keep, s[u][j], k * av[j]);
            acc[j] = fmaf(q, s[u][j], acc[j]);
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
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + kMemoryEps);
  float ss = 0.f;
  for (int p = threadIdx.x; p < P; p += THREADS) {
    float acc = 0.f;
    for (int q = 0; q < rows; ++q) acc += red[q * P + p];
    acc *= inv;
    sv[p] = acc;
    ss = fmaf(acc, acc, ss);
  }
  ss = block_sum(ss, part[1]);
  const float rstd = 1.f / sqrtf(ss / (float)P + eps);
  for (int p = threadIdx.x; p < L.pp; p += THREADS) {
    const int o = h * L.pp + p;
    cat[r * ldc + o] = from_f<T>(p < P ? sv[p] * rstd * L.gnorm[o] * sigmoid_as<T>(to_f(row[L.off_gg + o])) : 0.f);
  }
}

static int lanes_of(int p) {
  int l = 1;
  while (l < p && l < 32) l <<= 1;
  return l;
}

template <typename T>
static int launch_scan(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int seq0, int n_seq, cudaStream_t s) {
  static PerDeviceOnce once;
  auto floats = [&](int pc) { return (size_t)L.n * (pc + 1 + 2 * MS_T) + MS_T * pc + (size_t)(MS_THREADS / lanes_of(pc)) * pc; };
  int pc = L.p;
  while (pc > 1 && 4 * floats(pc) > 200 * 1024) pc = (pc + 1) / 2;
  const size_t smem = 4 * floats(pc);
  if (smem > 200 * 1024) return BB_ESIZE;
  const cudaError_t e = ensure_dyn_smem(once, hy_mlstm_scan_kernel<T>, 200 * 1024);
  if (e != cudaSuccess) return (int)e;
  for (int c0 = 0; c0 < L.p; c0 += pc)
    hy_mlstm_scan_kernel<T><<<dim3(n_seq, L.heads), MS_THREADS, smem, s>>>(
        L, static_cast<const T*>(w.proj), w.ld_proj, w.f32, w.ld_f32, static_cast<T*>(w.y), w.ld_y, b, seq0, c0, pc, c0 + pc >= L.p);
  return (int)cudaGetLastError();
}

template <typename T, int V, int THREADS>
static int launch_decode_v(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  static PerDeviceOnce once;
  const int rows = THREADS / lanes_of(L.p / V);
  const size_t smem = 4ull * (((L.p + 2 * L.n + 3) & ~3) + (size_t)rows * L.p);
  if (smem > 200 * 1024) return BB_ESIZE;
  if (smem > 40 * 1024) {
    const cudaError_t e = ensure_dyn_smem(once, hy_mlstm_decode_kernel<T, V, THREADS>, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  hy_mlstm_decode_kernel<T, V, THREADS><<<dim3(b.ns - b.ns_pre, L.heads), THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, w.f32, w.ld_f32, static_cast<T*>(w.cat), w.ld_cat, b, eps);
  return (int)cudaGetLastError();
}
template <typename T>
static int launch_decode(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  if (L.p % 4) return launch_decode_v<T, 1, 128>(L, w, b, eps, s);
  // large states, and few blocks: more threads share one
  return (long)L.n * L.p <= 128 * 128 && (long)(b.ns - b.ns_pre) * L.heads > 4 * sm_count()
             ? launch_decode_v<T, 4, 128>(L, w, b, eps, s)
             : launch_decode_v<T, 4, 256>(L, w, b, eps, s);
}

}  // namespace bb

using namespace bb;

// Log gates of the first n rows, in place of their raw values in w->f32.
BB_API int bb_hy_mlstm_gates(const BbHyCfg*, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  hy_mlstm_gates_kernel<<<(int)(((long)n * L->heads + 127) / 128), 128, 0, (cudaStream_t)stream>>>(*L, w->f32, w->ld_f32, n);
  return (int)cudaGetLastError();
}

// Sequences [seq0, seq0 + n_seq) of the step token by token, from the raw gates -> w->y.
BB_API int bb_hy_mlstm_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int seq0, int n_seq,
                            void* stream) {
  if (n_seq <= 0) return BB_OK;
  return c->dtype ? launch_scan<float>(*L, *w, *b, seq0, n_seq, (cudaStream_t)stream)
                  : launch_scan<__nv_bfloat16>(*L, *w, *b, seq0, n_seq, (cudaStream_t)stream);
}

// The decoded rows, norm and gate included -> w->cat; BB_ESIZE for heads the shared memory does not hold.
BB_API int bb_hy_mlstm_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->ns <= b->ns_pre) return BB_OK;
  return c->dtype ? launch_decode<float>(*L, *w, *b, c->eps, (cudaStream_t)stream)
                  : launch_decode<__nv_bfloat16>(*L, *w, *b, c->eps, (cudaStream_t)stream);
}

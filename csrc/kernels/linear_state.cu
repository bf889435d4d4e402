// Linear attention with a decaying state (fp32 state and recurrence, bf16 or fp32 projections).  Per head, with a decay
// per key channel,
//   S <- diag(decay) S + k v^T,   o = S^T q
// and the head's output is o over its root mean square, times a gain (or none) and the silu of a gate.  The decays are
// constants of the heads, or sigmoid(z)^root of a token's z; what is carried is decay - 1 (expm1 of the logarithm), so that
// a decay next to one keeps its rate.
//   hy_linear_scan    prompt portions that the chunked kernels (gla_tcgen05, ssd_tcgen05) do not cover: the state of a (sequence, head, value columns) in registers, four or more key
//                     channels times eight value columns to a thread; tokens come in tiles through shared memory
//   hy_linear_decode  one token per sequence: z, rotation, state, norm and gate in one kernel; the state is read and
//                     written once
//   hy_linear_post    norm and gate, where a head's columns were spread over blocks
// State of a head: [n][p].  A sequence at position 0 starts from zeros whatever its slot holds.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

// decay - 1 from z
__device__ __forceinline__ float decay_less(float z, float root) {
  return expm1f(-root * (fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))));
}

__device__ __forceinline__ void copy16_async(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// tokens of a tile, by the channels that its lanes cover
__host__ __device__ constexpr int scan_tokens(int wide) { return wide > 256 ? 8 : 16; }

// What a tile keeps in shared memory, in floats: raw inputs (two tiles), decays, keys and queries [tok][channels], values
// and outputs [tok][columns].
template <typename T>
struct ScanTile {
  int np, pc, pr;                // padded channels, columns of the block, columns as they are copied (a multiple of 8)
  bool z;
  __host__ __device__ int raw_row() const { return (2 * np + 2 * pr) * (int)sizeof(T) + (z ? 4 * np : 0); }   // bytes of a token
  __host__ __device__ size_t bytes(int wide) const {
    const int tok = scan_tokens(wide);
    return (size_t)2 * tok * raw_row() + 4ull * tok * (3 * wide + 2 * pc);
  }
};

// NG lanes share a column's channels, A channels each; 32 / NG groups of 8 columns to a warp.  FUSE: the block has all of a
// head's columns and finishes its rows (-> cat), else outputs go to y.  marks (may be null): of every (chunk of 128 tokens,
// head); pairs without any are left alone.
template <typename T, int NG, int A, bool FUSE>
__global__ void __launch_bounds__(256)
hy_linear_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const float* __restrict__ z,
                      int ldz, T* __restrict__ out, int ldo, const __grid_constant__ BbHyBatch b, int pc,
                      const int* __restrict__ marks, float eps) {
  extern __shared__ __align__(16) unsigned char ls_smem[];
  constexpr int NW = NG * A;                          // channels that the lanes cover
  constexpr int LS_TOK = scan_tokens(NW);
  const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * pc;
  if (marks) {
    const int n = (b.seq_row0[seq + 1] - b.seq_row0[seq] + 127) / 128, s0 = b.seq_row0[seq] / 128 + seq;
    bool any = false;
    for (int c = 0; c < n; ++c) any |= marks[(s0 + c) * L.heads + h] != 0;
    if (!any) return;
  }
  const int tid = threadIdx.x, nt_all = blockDim.x, lane = tid & 31, ng = lane % NG;
  const int col = ((tid >> 5) * (32 / NG) + lane / NG) * 8;        // first of the thread's columns in the block
  const int N = L.n, P = L.p;
  const ScanTile<T> tile{L.np, pc, min(pc, L.pp - c0), z != nullptr};
  const int raw_row = tile.raw_row(), np = L.np, pr = tile.pr;
  unsigned char* raw = ls_smem;
  float* s_w = reinterpret_cast<float*>(ls_smem + 2 * LS_TOK * raw_row);
  float *s_k = s_w + LS_TOK * NW, *s_q = s_k + LS_TOK * NW, *s_v = s_q + LS_TOK * NW, *s_o = s_v + LS_TOK * pc;
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1];
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * N * P;
  const bool fresh = b.seq_pos0[seq] == 0;

  // raw row of a token: k | q | v | gate (of this block's columns) | z
  const int ck = np * (int)sizeof(T) / 16, cv = pr * (int)sizeof(T) / 16, cz = tile.z ? np / 4 : 0, cr = 2 * ck + 2 * cv + cz;
  auto issue = [&](int t0, int buf) {
    const int nt = min(LS_TOK, r1 - t0);
    for (int i = tid; i < nt * cr; i += nt_all) {
      const int t = i / cr, c = i - t * cr;
      const T* row = proj + (size_t)(t0 + t) * ld;
      const void* src;
      if (c < ck) src = reinterpret_cast<const unsigned char*>(row + L.off_kk + h * np) + c * 16;
      else if (c < 2 * ck) src = reinterpret_cast<const unsigned char*>(row + L.off_q + h * np) + (c - ck) * 16;
      else if (c < 2 * ck + cv) src = reinterpret_cast<const unsigned char*>(row + L.off_vv + h * L.pp + c0) + (c - 2 * ck) * 16;
      else if (c < 2 * ck + 2 * cv) src = reinterpret_cast<const unsigned char*>(row + L.off_gg + h * L.pp + c0) + (c - 2 * ck - cv) * 16;
      else src = reinterpret_cast<const unsigned char*>(z + (size_t)(t0 + t) * ldz + h * np) + (c - 2 * ck - 2 * cv) * 16;
      copy16_async(raw + (size_t)(buf * LS_TOK + t) * raw_row + c * 16, src);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(r0, 0);

  float S[A][8];
#pragma unroll
  for (int i = 0; i < A; ++i) {
    const int n = (i / 4 * NG + ng) * 4 + i % 4;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int p = c0 + col + j;
      S[i][j] = !fresh && n < N && col + j < pc && p < P ? state[(size_t)n * P + p] : 0.f;
    }
  }
  const float keep = tile.z ? 0.f : L.keep_less[h];
  int buf = 0;
  for (int t0 = r0; t0 < r1; t0 += LS_TOK, buf ^= 1) {
    const int nt = min(LS_TOK, r1 - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                     // the tile is there, and the one before is done with
    if (t0 + LS_TOK < r1) issue(t0 + LS_TOK, buf ^ 1);
    const unsigned char* rb = raw + (size_t)buf * LS_TOK * raw_row;
    for (int i = tid; i < nt * NW; i += nt_all) {
      const int t = i / NW, n = i % NW;
      const T* kr = reinterpret_cast<const T*>(rb + (size_t)t * raw_row);
      const float* zr = reinterpret_cast<const float*>(kr + 2 * np + 2 * pr);
      const bool in = n < N;
      s_k[i] = in ? to_f(kr[n]) : 0.f;
      s_q[i] = in ? to_f(kr[np + n]) * L.q_scale : 0.f;
      s_w[i] = !in ? 0.f : (tile.z ? decay_less(zr[n] + L.w0[h * np + n], L.decay_root) : keep);
    }
    for (int i = tid; i < nt * pc; i += nt_all) {
      const int t = i / pc, p = i % pc;
      s_v[i] = p < pr ? to_f(reinterpret_cast<const T*>(rb + (size_t)t * raw_row)[2 * np + p]) : 0.f;
    }
    __syncthreads();
    if (col < pc) {
#pragma unroll 2
      for (int t = 0; t < nt; ++t) {
        float o[8], v[8];
        load8(s_v + t * pc + col, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] = 0.f;
#pragma unroll
        for (int a = 0; a < A / 4; ++a) {
          const int at = t * NW + (a * NG + ng) * 4;
          const float4 w4 = *reinterpret_cast<const float4*>(s_w + at), k4 = *reinterpret_cast<const float4*>(s_k + at),
                       q4 = *reinterpret_cast<const float4*>(s_q + at);
          const float w[4] = {w4.x, w4.y, w4.z, w4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              float& s = S[a * 4 + i][j];
              s = fmaf(k[i], v[j], fmaf(w[i], s, s));
              o[j] = fmaf(q[i], s, o[j]);
            }
        }
        // sum over the NG lanes; three steps leave one column to a lane
        const bool u2 = lane & 4, u1 = lane & 2, u0 = lane & 1;
        float x4[4], x2[2], x1;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float mine = u2 ? o[4 + j] : o[j], give = u2 ? o[j] : o[4 + j];
          x4[j] = mine + __shfl_xor_sync(0xffffffffu, give, 4);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float mine = u1 ? x4[2 + j] : x4[j], give = u1 ? x4[j] : x4[2 + j];
          x2[j] = mine + __shfl_xor_sync(0xffffffffu, give, 2);
        }
        x1 = (u0 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, u0 ? x2[0] : x2[1], 1);
        if (NG >= 16) x1 += __shfl_xor_sync(0xffffffffu, x1, 8);
        if (NG >= 32) x1 += __shfl_xor_sync(0xffffffffu, x1, 16);
        if (ng < 8) s_o[t * pc + col + (lane & 7)] = x1;
      }
    }
    __syncthreads();
    if constexpr (FUSE) {
      for (int t = tid >> 5; t < nt; t += nt_all >> 5) {
        const T* g = reinterpret_cast<const T*>(rb + (size_t)t * raw_row) + 2 * np + pr;
        float ss = 0.f;
        for (int p = lane; p < P; p += 32) ss = fmaf(s_o[t * pc + p], s_o[t * pc + p], ss);
        ss = warp_sum(ss);
        const float rstd = 1.f / sqrtf(ss / (float)P + eps);
        T* dst = out + (size_t)(t0 + t) * ldo + h * L.pp;
        for (int p = lane; p < L.pp; p += 32) {
          float x = 0.f;
          if (p < P) {
            x = s_o[t * pc + p] * rstd * silu_as<T>(to_f(g[p]));
            if (L.gnorm) x *= L.gnorm[h * L.pp + p];
          }
          dst[p] = from_f<T>(x);
        }
      }
    } else {
      for (int i = tid; i < nt * pr; i += nt_all) {
        const int t = i / pr, p = i % pr;
        out[(size_t)(t0 + t) * ldo + h * L.pp + c0 + p] = from_f<T>(c0 + p < P ? s_o[t * pc + p] : 0.f);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < A; ++i) {
    const int n = (i / 4 * NG + ng) * 4 + i % 4;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int p = c0 + col + j;
      if (n < N && col + j < pc && p < P) state[(size_t)n * P + p] = S[i][j];
    }
  }
}

// V: state elements of a lane (4: 16-byte accesses, p % 4 == 0; 1: any p).
template <typename T, int V, int THREADS>
__global__ void __launch_bounds__(THREADS)
hy_linear_decode_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, T* __restrict__ cat, int ldc,
                        const __grid_constant__ BbHyBatch b, float eps) {
  extern __shared__ float sm[];
  const int seq = b.ns_pre + blockIdx.x, h = blockIdx.y, N = L.n, P = L.p;
  const size_t r = b.n_pre + blockIdx.x;
  float* sv = sm;              // [P], then the outputs
  float *sq = sv + P, *sk = sq + N, *sw = sk + N;      // [N] each
  float* red = sm + ((P + 3 * N + 3) & ~3);            // [rows][P]
  __shared__ float part[32];
  const T* row = proj + r * ld;
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * N * P;
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
  const int pos = b.pos[r];
  const bool fresh = pos == 0;
  fetch(nr, lane);
  for (int p = threadIdx.x; p < P; p += THREADS) sv[p] = to_f(row[L.off_vv + h * L.pp + p]);
  for (int d = threadIdx.x; d < N; d += THREADS) {
    const T *qr = row + L.off_q + h * L.np, *kr = row + L.off_kk + h * L.np;
    float q = to_f(qr[d]), k = to_f(kr[d]);
    if (d < L.rot) {             // neighbouring pairs
      const size_t t = (size_t)pos * (L.rot >> 1) + (d >> 1);
      const float co = L.cos_t[t], si = d & 1 ? L.sin_t[t] : -L.sin_t[t];
      q = fmaf(q, co, to_f(qr[d ^ 1]) * si);
      k = fmaf(k, co, to_f(kr[d ^ 1]) * si);
    }
    sq[d] = q * L.q_scale;
    sk[d] = k;
    if (L.w2.w) {
      const T *w = static_cast<const T*>(L.w2.w) + (size_t)(h * L.np + d) * L.wrp, *a = row + L.off_w1;
      float z = L.w0[h * L.np + d];
      for (int i = 0; i < L.wrp; i += 8) {
        float f[8], g[8];
        load8(w + i, f);
        load8(a + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) z = fmaf(f[j], g[j], z);
      }
      sw[d] = decay_less(z, L.decay_root);
    } else {
      sw[d] = L.keep_less[h];
    }
  }
  __syncthreads();
  for (int p = lane; p < pv; p += lanes) {
    float v[V], acc[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      v[j] = sv[p * V + j];
      acc[j] = 0.f;
    }
    for (int n0 = nr; n0 < N; n0 += U * rows) {
      if (p != lane || n0 != nr) fetch(n0, p);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int n = n0 + u * rows;
        if (n < N) {
          const float k = sk[n], q = sq[n], w = sw[n];
#pragma unroll
          for (int j = 0; j < V; ++j) {      // a fresh sequence ignores whatever its slot holds (it may not be a number)
            s[u][j] = fresh ? k * v[j] : fmaf(k, v[j], fmaf(w, s[u][j], s[u][j]));
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
  float ss = 0.f;
  for (int p = threadIdx.x; p < P; p += THREADS) {
    float acc = 0.f;
    for (int q = 0; q < rows; ++q) acc += red[q * P + p];
    sv[p] = acc;
    ss = fmaf(acc, acc, ss);
  }
  ss = block_sum(ss, part);
  const float rstd = 1.f / sqrtf(ss / (float)P + eps);
  for (int p = threadIdx.x; p < L.pp; p += THREADS) {
    const int o = h * L.pp + p;
    float x = 0.f;
    if (p < P) {
      x = sv[p] * rstd * silu_as<T>(to_f(row[L.off_gg + o]));
      if (L.gnorm) x *= L.gnorm[o];
    }
    cat[r * ldc + o] = from_f<T>(x);
  }
}

constexpr int LP_THREADS = 256;

// `lanes` threads (a power of two up to a warp) share a head.
template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
hy_linear_post_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ y, int ldy,
                      T* __restrict__ cat, int ldc, int lanes, float eps) {
  const size_t r = blockIdx.x;
  const int lane = threadIdx.x % lanes, groups = LP_THREADS / lanes, vecs = L.pp / 8;
  for (int h0 = 0; h0 < L.heads; h0 += groups) {
    const int h = h0 + threadIdx.x / lanes;
    const bool live = h < L.heads;
    float f[8], g[8], ss = 0.f;
    auto load = [&](int v) {
      load8(y + r * ldy + h * L.pp + v * 8, f);
      load8(proj + r * ld + L.off_gg + h * L.pp + v * 8, g);
    };
    for (int v = lane; live && v < vecs; v += lanes) {
      load(v);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rstd = 1.f / sqrtf(ss / (float)L.p + eps);
    for (int v = lane; live && v < vecs; v += lanes) {
      if (vecs > lanes) load(v);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= rstd * silu_as<T>(g[j]);
      if (L.gnorm) {
        load8(L.gnorm + h * L.pp + v * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= g[j];
      }
      store8(cat + r * ldc + h * L.pp + v * 8, f);
    }
  }
}

template <typename T>
static int launch_post(const BbHyLayer& L, const BbHyWork& w, int rows, float eps, cudaStream_t s) {
  if (rows <= 0) return BB_OK;
  int lanes = 1;
  while (lanes < L.pp / 8 && lanes < 32) lanes <<= 1;
  hy_linear_post_kernel<T><<<rows, LP_THREADS, 0, s>>>(L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.y), w.ld_y,
                                                       static_cast<T*>(w.cat), w.ld_cat, lanes, eps);
  return (int)cudaGetLastError();
}

template <typename T, int NG, int A>
static int launch_scan_n(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, const float* z, const int* marks,
                         float eps, cudaStream_t s) {
  static PerDeviceOnce once, once_fused;
  constexpr int LIMIT = 200 * 1024;
  cudaError_t e = ensure_dyn_smem(once, hy_linear_scan_kernel<T, NG, A, false>, LIMIT);
  if (e != cudaSuccess) return (int)e;
  e = ensure_dyn_smem(once_fused, hy_linear_scan_kernel<T, NG, A, true>, LIMIT);
  if (e != cudaSuccess) return (int)e;
  // columns of a block: up to eight warps, as few parts of a head as keep the machine's warps busy
  constexpr int WARP_COLS = 32 / NG * 8;
  const long pairs = (long)b.ns_pre * L.heads;
  const int sms = sm_count();
  int pc = 0;
  long best = 0;
  for (int warps = 8; warps >= 1; warps >>= 1) {
    const int c = warps * WARP_COLS, parts = (L.p + c - 1) / c, used = parts > 1 ? warps : (L.p + WARP_COLS - 1) / WARP_COLS;
    if (marks && parts > 1) continue;                          // (the other pairs' rows are finished)
    if (ScanTile<T>{L.np, parts > 1 ? c : used * WARP_COLS, c, z != nullptr}.bytes(NG * A) > LIMIT) continue;
    long cost = (pairs * parts + sms - 1) / sms * used;       // warps that follow one another on an SM
    cost = (cost < 4 ? 4 : cost) * 16 + (parts > 1 ? 4 : 0);  // (a split head takes another launch)
    if (!pc || cost < best) {
      pc = parts > 1 ? c : used * WARP_COLS;
      best = cost;
    }
  }
  if (!pc) return BB_ESIZE;
  const int parts = (L.p + pc - 1) / pc, threads = pc / WARP_COLS * 32;
  const size_t smem = ScanTile<T>{L.np, pc, pc, z != nullptr}.bytes(NG * A);
  const T* proj = static_cast<const T*>(w.proj);
  const dim3 grid(b.ns_pre, L.heads, parts);
  if (parts == 1) {
    hy_linear_scan_kernel<T, NG, A, true><<<grid, threads, smem, s>>>(L, proj, w.ld_proj, z, w.ld_f32, static_cast<T*>(w.cat),
                                                                      w.ld_cat, b, pc, marks, eps);
    return (int)cudaGetLastError();
  }
  hy_linear_scan_kernel<T, NG, A, false><<<grid, threads, smem, s>>>(L, proj, w.ld_proj, z, w.ld_f32, static_cast<T*>(w.y),
                                                                     w.ld_y, b, pc, marks, eps);
  e = cudaGetLastError();
  return e != cudaSuccess ? (int)e : launch_post<T>(L, w, b.n_pre, eps, s);
}
template <typename T>
static int launch_scan(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, const float* z, const int* marks, float eps,
                       cudaStream_t s) {
  if (b.ns_pre <= 0) return BB_OK;
  if (L.n <= 32) return launch_scan_n<T, 8, 4>(L, w, b, z, marks, eps, s);
  if (L.n <= 64) return launch_scan_n<T, 16, 4>(L, w, b, z, marks, eps, s);
  if (L.n <= 128) return launch_scan_n<T, 32, 4>(L, w, b, z, marks, eps, s);
  if (L.n <= 256) return launch_scan_n<T, 32, 8>(L, w, b, z, marks, eps, s);
  return L.n <= 512 ? launch_scan_n<T, 32, 16>(L, w, b, z, marks, eps, s) : BB_ESIZE;
}

static int lanes_of(int p) {
  int l = 1;
  while (l < p && l < 32) l <<= 1;
  return l;
}
template <typename T, int V, int THREADS>
static int launch_decode_v(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, float eps, cudaStream_t s) {
  static PerDeviceOnce once;
  const int rows = THREADS / lanes_of(L.p / V);
  const size_t smem = 4ull * (((L.p + 3 * L.n + 3) & ~3) + (size_t)rows * L.p);
  if (smem > 200 * 1024) return BB_ESIZE;
  if (smem > 40 * 1024) {
    const cudaError_t e = ensure_dyn_smem(once, hy_linear_decode_kernel<T, V, THREADS>, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  hy_linear_decode_kernel<T, V, THREADS><<<dim3(b.ns - b.ns_pre, L.heads), THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<T*>(w.cat), w.ld_cat, b, eps);
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

// The prompt portions token by token: recurrence, norm and gate -> w->cat.  Queries and keys are rotated; z of a token in
// w->f32 where decays are not constant.  `marked`: only the pairs that bb_gla_chunk has marked.
BB_API int bb_hy_linear_scan(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int marked, void* stream) {
  const float* z = L->w2.w ? w->f32 : nullptr;
  const int* marks = marked ? w->chunk_flags : nullptr;
  cudaStream_t s = (cudaStream_t)stream;
  return c->dtype ? launch_scan<float>(*L, *w, *b, z, marks, c->eps, s)
                  : launch_scan<__nv_bfloat16>(*L, *w, *b, z, marks, c->eps, s);
}

// The single tokens -> w->cat; BB_ESIZE for heads the shared memory does not hold.
BB_API int bb_hy_linear_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->ns <= b->ns_pre) return BB_OK;
  return c->dtype ? launch_decode<float>(*L, *w, *b, c->eps, (cudaStream_t)stream)
                  : launch_decode<__nv_bfloat16>(*L, *w, *b, c->eps, (cudaStream_t)stream);
}

// Norm and gate of the first `rows` rows of w->y -> w->cat.
BB_API int bb_hy_linear_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int rows, void* stream) {
  return c->dtype ? launch_post<float>(*L, *w, rows, c->eps, (cudaStream_t)stream)
                  : launch_post<__nv_bfloat16>(*L, *w, rows, c->eps, (cudaStream_t)stream);
}

// Row kernels of the hybrid decoder, one block per token row, fp32 arithmetic, bf16 or fp32 storage:
//   hy_embed_norm   embedding row -> RMS norm -> fp32 residual stream
//   hy_norm         residual row (optionally picked by an index list) -> RMS norm -> projection input
//   hy_attn_post    after the fused input projection of an attention layer: RMS norm over the whole q and
//                   the whole k, partial rotation, value mixing with an earlier layer, K/V written
//                   straight into the sequence's page, and the layer's gated feed-forward product
//   hy_start        a layer's start: embedding (scaled, plus a learned vector per position) or residual row, plus
//                   the weighted outputs of the row's experts of the layer before -> residual stream (plus the
//                   biases that this layer will add) and RMS norm -> projection input
//   hy_kv_post      attention without norms: biases, queries in place, K/V into the page, feed-forward product
//   hy_glu          the gated feed-forward product alone
//   hy_mamba_post   after the state-space recurrence: silu(z) gate, grouped RMS norm, the last raw inputs
//                   of the convolution into the sequence's state slot, and the feed-forward product
// The two "post" kernels write the mixer's (or only the feed-forward's) part of the row that the fused
// output projection multiplies, so a layer's two sublayers share one output GEMM.
#include "../common/host.hpp"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int ROW_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
hy_embed_norm_kernel(const int* __restrict__ tok, const T* __restrict__ emb, const float* __restrict__ w,
                     float* __restrict__ x, int d, int dp, int vocab, float eps) {
  __shared__ float buf[32];
  const int r = blockIdx.x;
  int id = tok[r];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* e = emb + (size_t)id * dp;
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < dp; i += blockDim.x * 8) {
    float f[8];
    load8(e + i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
  }
  ss = block_sum(ss, buf);
  const float rstd = 1.f / sqrtf(ss / (float)d + eps);
  for (int i = threadIdx.x * 8; i < dp; i += blockDim.x * 8) {
    float f[8], g[8];
    load8(e + i, f);
    load8(w + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = f[j] * rstd * g[j];
    store8(x + (size_t)r * dp + i, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
hy_norm_kernel(const float* __restrict__ x, const int* __restrict__ rows, const float* __restrict__ w,
               T* __restrict__ h, int d, int dp, float eps) {
  __shared__ float buf[32];
  const float* xr = x + (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * dp;
  constexpr int KEEP = 2;   // vectors of a row that stay in registers (rows up to 4096 wide)
  float v[KEEP][8];
  float ss = 0.f;
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (threadIdx.x + t * blockDim.x) * 8;
    if (i < dp) {
      load8(xr + i, v[t]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[t][j] * v[t][j];
    }
  }
  for (int i = (threadIdx.x + KEEP * blockDim.x) * 8; i < dp; i += blockDim.x * 8) {
    float f[8];
    load8(xr + i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
  }
  ss = block_sum(ss, buf);
  const float rstd = 1.f / sqrtf(ss / (float)d + eps);
  T* hr = h + (size_t)blockIdx.x * dp;
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (threadIdx.x + t * blockDim.x) * 8;
    if (i < dp) {
      float g[8];
      load8(w + i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] *= v[t][j] * rstd;
      store8(hr + i, g);
    }
  }
  for (int i = (threadIdx.x + KEEP * blockDim.x) * 8; i < dp; i += blockDim.x * 8) {
    float f[8], g[8];
    load8(xr + i, f);
    load8(w + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = f[j] * rstd * g[j];
    store8(hr + i, f);
  }
}

// Row vectors beyond KEEP a thread go through the residual stream where it is written (a thread reads back what it
// wrote).  Block 0 clears the expert counts of the layer that starts.
struct StartArgs {
  float* x;
  const int *rows, *tok, *pos;     // rows: residual row of every block (null: its own)
  const void *emb, *pos_tab;
  float emb_scale;
  int vocab, max_pos, embed;       // embed: rows come from the embedding
  const void* ex_out;              // experts of the layer before (top = 0: none)
  const int* pair_row;
  const float* pair_w;
  int top;
  const float *w, *bias;           // gain; bias added to the residual row (null: none)
  int write, d, dp;                // write: the residual row changes
  float eps;
  int *counts, n_counts;
  float* trace;
};

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS, 4)
hy_start_kernel(const __grid_constant__ StartArgs a, T* __restrict__ h) {
  __shared__ float buf[32];
  const int r = a.rows ? a.rows[blockIdx.x] : (int)blockIdx.x;
  float* xr = a.x + (size_t)r * a.dp;
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e < a.n_counts; e += ROW_THREADS) a.counts[e] = 0;
  const T *er = nullptr, *pr = nullptr;
  if (a.embed) {
    er = static_cast<const T*>(a.emb) + (size_t)min(max(a.tok[r], 0), a.vocab - 1) * a.dp;
    if (a.pos_tab) pr = static_cast<const T*>(a.pos_tab) + (size_t)min(max(a.pos[r], 0), a.max_pos - 1) * a.dp;
  }
  const int* prow = a.pair_row + (size_t)r * a.top;
  const float* pw = a.pair_w + (size_t)r * a.top;
  auto fetch = [&](int i, float (&f)[8]) {
    if (er) {
      load8(er + i, f);
      float p[8] = {};
      if (pr) load8(pr + i, p);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = fmaf(f[j], a.emb_scale, p[j]);
    } else {
      load8(xr + i, f);
    }
    if (a.top > 0) {
      float y[8] = {};
#pragma unroll 4
      for (int s = 0; s < a.top; ++s) {
        float g[8];
        load8(static_cast<const T*>(a.ex_out) + (size_t)prow[s] * a.dp + i, g);
        const float w = pw[s];
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] = fmaf(w, g[j], y[j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] += y[j];
    }
  };
  constexpr int KEEP = 2;
  float v[KEEP][8];
  float ss = 0.f;
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (threadIdx.x + t * ROW_THREADS) * 8;
    if (i < a.dp) {
      fetch(i, v[t]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[t][j] * v[t][j];
    }
  }
  for (int i = (threadIdx.x + KEEP * ROW_THREADS) * 8; i < a.dp; i += ROW_THREADS * 8) {
    float f[8];
    fetch(i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    if (a.write) store8(xr + i, f);
  }
  ss = block_sum(ss, buf);
  const float rstd = 1.f / sqrtf(ss / (float)a.d + a.eps);
  T* hr = h + (size_t)blockIdx.x * a.dp;
  auto emit = [&](int i, float (&f)[8]) {
    if (a.trace) store8(a.trace + (size_t)r * a.dp + i, f);
    float g[8];
    load8(a.w + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] *= f[j] * rstd;
    store8(hr + i, g);
    if (a.write) {
      if (a.bias) {
        load8(a.bias + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] += g[j];
      }
      store8(xr + i, f);
    }
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = (threadIdx.x + t * ROW_THREADS) * 8;
    if (i < a.dp) emit(i, v[t]);
  }
  for (int i = (threadIdx.x + KEEP * ROW_THREADS) * 8; i < a.dp; i += ROW_THREADS * 8) {
    float f[8];
    if (a.write) load8(xr + i, f);
    else fetch(i, f);
    emit(i, f);
  }
}

// Blocks of a "post" launch: blockIdx.y = 0 is the row's mixer part, every further one GLU_COLS columns of
// its feed-forward product (GLU_VECS vectors of a thread, all asked for before the first is used).
constexpr int GLU_VECS = 3;
constexpr int GLU_COLS = ROW_THREADS * 8 * GLU_VECS;

template <typename T, int KIND = 0>
__device__ __forceinline__ void glu_part(const BbHyLayer& L, const T* row, T* crow, int part) {
  struct alignas(sizeof(T) * 8) Raw {
    T v[8];
  };
  const int n = (L.ff + 7) & ~7, i0 = part * GLU_COLS + threadIdx.x * 8;
  Raw g[GLU_VECS], u[GLU_VECS];
#pragma unroll
  for (int t = 0; t < GLU_VECS; ++t) {
    const int i = i0 + t * ROW_THREADS * 8;
    if (i < n) {
      g[t] = *reinterpret_cast<const Raw*>(row + L.off_gate + i);
      u[t] = *reinterpret_cast<const Raw*>(row + L.off_up + i);
    }
  }
#pragma unroll
  for (int t = 0; t < GLU_VECS; ++t) {
    const int i = i0 + t * ROW_THREADS * 8;
    if (i < n) {
      float f[8];
      if constexpr (KIND == 0) {
#pragma unroll
        for (int j = 0; j < 8; ++j)
          f[j] = clamped_glu_as<T>(to_f(g[t].v[j]), to_f(u[t].v[j]), L.glu_limit, L.glu_alpha, L.glu_shift);
      } else {                       // biases are zero in the padding, and so is the product
        float gb[8], ub[8];
        load8(L.gate_b + i, gb);
        load8(L.up_b + i, ub);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = gelu_as<T>(to_f(g[t].v[j]) + gb[j]) * (to_f(u[t].v[j]) + ub[j]);
      }
      store8(crow + L.off_act + i, f);
    }
  }
}

template <typename T, int KIND>
__global__ void __launch_bounds__(ROW_THREADS, sizeof(T) == 2 ? 5 : 4)
hy_glu_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, T* __restrict__ cat, int ldc) {
  glu_part<T, KIND>(L, proj + (size_t)blockIdx.x * ld, cat + (size_t)blockIdx.x * ldc, blockIdx.y);
}

// blockIdx.y = 0: queries, keys and values of a row; further blocks its feed-forward product.
template <typename T, int KIND>
__global__ void __launch_bounds__(ROW_THREADS, sizeof(T) == 2 ? 5 : 4)
hy_kv_post_kernel(const __grid_constant__ BbHyLayer L, T* __restrict__ proj, int ld, T* __restrict__ cat, int ldc,
                  const int* __restrict__ pos_, const int* __restrict__ row_seq, const int* __restrict__ tables,
                  int max_blocks, int bs) {
  const int r = blockIdx.x;
  T* row = proj + (size_t)r * ld;
  if (blockIdx.y > 0) {
    glu_part<T, KIND>(L, row, cat + (size_t)r * ldc, blockIdx.y - 1);
    return;
  }
  const int nq = L.q_b ? L.hq * L.dkp : 0, nk = L.hk * L.dkp, nv = L.hk * L.dvp;
  const int pos = pos_[r], blk = tables[(size_t)row_seq[r] * max_blocks + pos / bs], off = pos % bs;
  for (int i = threadIdx.x * 8; i < nq + nk + nv; i += ROW_THREADS * 8) {
    const int part = i < nq ? 0 : (i < nq + nk ? 1 : 2), o = part == 0 ? i : (part == 1 ? i - nq : i - nq - nk);
    T* src = row + (part == 0 ? L.off_q : (part == 1 ? L.off_k : L.off_v)) + o;
    float f[8];
    load8(src, f);
    if (L.q_b) {
      float bias[8];
      load8((part == 0 ? L.q_b : (part == 1 ? L.k_b : L.v_b)) + o, bias);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] += bias[j];
    }
    if (part == 0) {
      store8(src, f);
    } else {
      const int size = part == 1 ? L.dkp : L.dvp, h = o / size;
      store8(static_cast<T*>(part == 1 ? L.kc : L.vc) + (((size_t)blk * L.hk + h) * bs + off) * size + (o - h * size), f);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS, sizeof(T) == 2 ? 5 : 4)
hy_attn_post_kernel(const __grid_constant__ BbHyLayer L, T* __restrict__ proj, int ld, T* __restrict__ cat, int ldc,
                    T* __restrict__ v_first, int ldv, const int* __restrict__ pos_, const int* __restrict__ row_seq,
                    const int* __restrict__ tables, int max_blocks, int bs, float eps) {
  extern __shared__ __align__(16) float s_row[];   // q | k of the row, times their gains
  __shared__ float buf[2][32];
  const int r = blockIdx.x;
  T* row = proj + (size_t)r * ld;
  if (blockIdx.y > 0) {
    glu_part(L, row, cat + (size_t)r * ldc, blockIdx.y - 1);
    return;
  }
  const int nq = L.hq * L.dkp, nk = L.hk * L.dkp, nv = L.hk * L.dvp;
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x * 8; i < nq + nk; i += ROW_THREADS * 8) {
    float f[8], g[8];
    const bool is_q = i < nq;
    load8(is_q ? row + L.off_q + i : row + L.off_k + (i - nq), f);
    load8(is_q ? L.q_norm + i : L.k_norm + (i - nq), g);
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      s += f[j] * f[j];
      g[j] *= f[j];
    }
    store8(s_row + i, g);
    if (is_q) ssq += s; else ssk += s;
  }
  const int pos = pos_[r], seq = row_seq[r];
  const int blk = tables[(size_t)seq * max_blocks + pos / bs], off = pos % bs;
  ssq = block_sum(ssq, buf[0]);
  ssk = block_sum(ssk, buf[1]);    // (its barrier also orders the row in shared memory)
  const float rq = 1.f / sqrtf(ssq / (float)(L.hq * L.dk) + eps);
  const float rk = 1.f / sqrtf(ssk / (float)(L.hk * L.dk) + eps);
  const int half = L.rot >> 1;
  const float* ct = L.cos_t + (size_t)pos * half;
  const float* st = L.sin_t + (size_t)pos * half;
  T* kc = static_cast<T*>(L.kc);
  T* vc = static_cast<T*>(L.vc);
  for (int i = threadIdx.x * 8; i < nq + nk; i += ROW_THREADS * 8) {
    const bool is_q = i < nq;
    const int h = (is_q ? i : i - nq) / L.dkp, d0 = (is_q ? i : i - nq) - h * L.dkp;
    const float rs = is_q ? rq : rk;
    float f[8];
    load8(s_row + i, f);
    if ((half & 7) == 0) {           // a vector lies in one half of the rotated part, or past it
      if (d0 < L.rot) {
        const bool lo = d0 < half;
        float g[8], c[8], sn[8];
        load8(s_row + (lo ? i + half : i - half), g);
        load8(ct + (lo ? d0 : d0 - half), c);
        load8(st + (lo ? d0 : d0 - half), sn);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = lo ? f[j] * c[j] - g[j] * sn[j] : f[j] * c[j] + g[j] * sn[j];
      }
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int d = d0 + j, e = i + j;
        if (d < half) f[j] = f[j] * ct[d] - s_row[e + half] * st[d];
        else if (d < L.rot) f[j] = f[j] * ct[d - half] + s_row[e - half] * st[d - half];
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= rs;
    if (is_q) store8(row + L.off_q + i, f);
    else store8(kc + (((size_t)blk * L.hk + h) * bs + off) * L.dkp + d0, f);
  }
  for (int i = threadIdx.x * 8; i < nv; i += ROW_THREADS * 8) {
    float f[8];
    load8(row + L.off_v + i, f);
    T* vf = v_first + (size_t)r * ldv + i;
    if (L.v_role == 1) store8(vf, f);
    if (L.v_role == 2) {
      float g[8];
      load8(vf, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = (1.f - L.vmix) * f[j] + L.vmix * g[j];
    }
    const int h = i / L.dvp, d0 = i - h * L.dvp;
    store8(vc + (((size_t)blk * L.hk + h) * bs + off) * L.dvp + d0, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS, sizeof(T) == 2 ? 5 : 4)
hy_mamba_post_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ y,
                     int ldy, T* __restrict__ cat, int ldc, const int* __restrict__ pos_,
                     const int* __restrict__ row_seq, const int* __restrict__ seq_ctx,
                     const int* __restrict__ seq_slot, float eps) {
  extern __shared__ __align__(16) float s_row[];   // gated row, then one 1/rms per part
  float* s_rstd = s_row + L.innerp;
  __shared__ float part[ROW_THREADS / 32];
  const int r = blockIdx.x;
  const T* row = proj + (size_t)r * ld;
  if (blockIdx.y > 0) {
    glu_part(L, row, cat + (size_t)r * ldc, blockIdx.y - 1);
    return;
  }
  for (int i = threadIdx.x * 8; i < L.innerp; i += blockDim.x * 8) {
    float f[8], z[8];
    load8(y + (size_t)r * ldy + i, f);
    load8(row + L.off_z + i, z);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = i + j < L.inner ? f[j] * silu_as<T>(z[j]) : 0.f;
    store8(s_row + i, f);
  }
  __syncthreads();
  // one root mean square per part: with few parts several warps share one, with many a warp takes several
  const int ng = L.norm_groups, len = L.inner / ng;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = ROW_THREADS / 32;
  const int per = ng < nw ? nw / ng : 1;         // warps of a part
  for (int g0 = 0; g0 < ng; g0 += nw / per) {
    const int g = g0 + warp / per, sub = warp % per;
    float s = 0.f;
    if (g < ng && warp < (nw / per) * per)
      if ((len & 3) == 0)
        for (int i = (sub * 32 + lane) * 4; i < len; i += per * 128) {
          const float4 v = *reinterpret_cast<const float4*>(s_row + g * len + i);
          s += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
      else
        for (int i = sub * 32 + lane; i < len; i += per * 32) s += s_row[g * len + i] * s_row[g * len + i];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) part[warp] = s;
    __syncthreads();
    if (threadIdx.x < nw / per && g0 + threadIdx.x < ng) {
      float t = 0.f;
      for (int w = 0; w < per; ++w) t += part[threadIdx.x * per + w];
      s_rstd[g0 + threadIdx.x] = 1.f / sqrtf(t / (float)len + eps);
    }
    __syncthreads();
  }
  T* crow = cat + (size_t)r * ldc;
  for (int i = threadIdx.x * 8; i < L.innerp; i += blockDim.x * 8) {
    float f[8], w[8];
    load8(L.gnorm + i, w);           // zero past the last channel
    load8(s_row + i, f);
    if ((len & 7) == 0) {
      const float rs = s_rstd[min(i / len, ng - 1)];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= rs * w[j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= s_rstd[min((i + j) / len, ng - 1)] * w[j];
    }
    store8(crow + i, f);
  }
  // the last taps - 1 raw inputs of the sequence go to its slot (their ring places were read, if at all,
  // by the convolution that ran before this kernel)
  const int seq = row_seq[r], pos = pos_[r], keep = L.taps - 1;
  if (keep > 0 && pos >= seq_ctx[seq] - keep) {
    T* ring = static_cast<T*>(L.conv_state) + ((size_t)seq_slot[seq] * keep + pos % keep) * L.chp;
    for (int i = threadIdx.x * 8; i < L.chp; i += blockDim.x * 8) {
      float f[8];
      load8(row + L.off_xbc + i, f);
      store8(ring + i, f);
    }
  }
}

template <typename T>
static int launch_embed_norm(const BbHyCfg& c, const int* tok, float* x, int n, cudaStream_t s) {
  hy_embed_norm_kernel<T><<<n, ROW_THREADS, 0, s>>>(tok, static_cast<const T*>(c.embed), c.embed_norm, x, c.width,
                                                    c.dp, c.vocab, c.eps);
  return (int)cudaGetLastError();
}

// shared memory above the default 48 KB has to be asked for (once per device and kernel)
template <typename K>
static int row_smem(PerDeviceOnce& once, K kernel, size_t bytes) {
  if (bytes <= 40 * 1024) return BB_OK;
  if (bytes > 200 * 1024) return BB_ESIZE;
  return (int)ensure_dyn_smem(once, kernel, 200 * 1024);
}

template <typename T>
static int launch_attn_post(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once;
  const size_t smem = (size_t)(L.hq + L.hk) * L.dkp * 4;
  const int rc = row_smem(once, hy_attn_post_kernel<T>, smem);
  if (rc) return rc;
  hy_attn_post_kernel<T><<<dim3(b.n, 1 + (L.ff + GLU_COLS - 1) / GLU_COLS), ROW_THREADS, smem, s>>>(
      L, static_cast<T*>(w.proj), w.ld_proj, static_cast<T*>(w.cat), w.ld_cat, static_cast<T*>(w.v_first), w.ld_v,
      b.pos, b.row_seq, b.tables, b.max_blocks, c.block_size, c.eps);
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_mamba_post(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once;
  const size_t smem = (size_t)(L.innerp + L.norm_groups) * 4;
  const int rc = row_smem(once, hy_mamba_post_kernel<T>, smem);
  if (rc) return rc;
  hy_mamba_post_kernel<T><<<dim3(b.n, 1 + (L.ff + GLU_COLS - 1) / GLU_COLS), ROW_THREADS, smem, s>>>(
      L, static_cast<const T*>(w.proj), w.ld_proj, static_cast<const T*>(w.y), w.ld_y, static_cast<T*>(w.cat), w.ld_cat,
      b.pos, b.row_seq, b.seq_ctx, b.seq_slot, c.eps);
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_kv_post(const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  const dim3 grid(b.n, 1 + (L.ff + GLU_COLS - 1) / GLU_COLS);
  T *proj = static_cast<T*>(w.proj), *cat = static_cast<T*>(w.cat);
  if (L.glu_kind)
    hy_kv_post_kernel<T, 1><<<grid, ROW_THREADS, 0, s>>>(L, proj, w.ld_proj, cat, w.ld_cat, b.pos, b.row_seq, b.tables,
                                                         b.max_blocks, c.block_size);
  else
    hy_kv_post_kernel<T, 0><<<grid, ROW_THREADS, 0, s>>>(L, proj, w.ld_proj, cat, w.ld_cat, b.pos, b.row_seq, b.tables,
                                                         b.max_blocks, c.block_size);
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_glu(const BbHyLayer& L, const BbHyWork& w, int n, cudaStream_t s) {
  const dim3 grid(n, (L.ff + GLU_COLS - 1) / GLU_COLS);
  const T* proj = static_cast<const T*>(w.proj);
  T* cat = static_cast<T*>(w.cat);
  if (L.glu_kind) hy_glu_kernel<T, 1><<<grid, ROW_THREADS, 0, s>>>(L, proj, w.ld_proj, cat, w.ld_cat);
  else hy_glu_kernel<T, 0><<<grid, ROW_THREADS, 0, s>>>(L, proj, w.ld_proj, cat, w.ld_cat);
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

BB_API int bb_hy_embed_norm(const BbHyCfg* c, const int* tok, float* x, int n, void* stream) {
  if (n <= 0) return BB_EARG;
  return c->dtype ? launch_embed_norm<float>(*c, tok, x, n, (cudaStream_t)stream)
                  : launch_embed_norm<__nv_bfloat16>(*c, tok, x, n, (cudaStream_t)stream);
}

// h[i] = RMS norm of residual row rows[i] (i when rows is null) times the gain w.
BB_API int bb_hy_norm(int dtype, const float* x, const int* rows, const float* w, void* h, int n, int d, int dp,
                      float eps, void* stream) {
  if (n <= 0 || dp % 8) return BB_EARG;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype) hy_norm_kernel<float><<<n, ROW_THREADS, 0, s>>>(x, rows, w, static_cast<float*>(h), d, dp, eps);
  else hy_norm_kernel<__nv_bfloat16><<<n, ROW_THREADS, 0, s>>>(x, rows, w, static_cast<__nv_bfloat16*>(h), d, dp, eps);
  return (int)cudaGetLastError();
}

BB_API int bb_hy_attn_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? launch_attn_post<float>(*c, *L, *w, *b, (cudaStream_t)stream)
                  : launch_attn_post<__nv_bfloat16>(*c, *L, *w, *b, (cudaStream_t)stream);
}

BB_API int bb_hy_mamba_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? launch_mamba_post<float>(*c, *L, *w, *b, (cudaStream_t)stream)
                  : launch_mamba_post<__nv_bfloat16>(*c, *L, *w, *b, (cudaStream_t)stream);
}

// Start of layer li (li = n_layers: the rows whose logits are asked for -> hn).  `all`: every row, even past the
// last layer.
BB_API int bb_hy_start(const BbHyCfg* c, int li, const BbHyWork* w, const BbHyBatch* b, int all, float* trace, void* stream) {
  const BbHyLayer* L = li < c->n_layers ? c->layers + li : nullptr;
  const BbHyLayer* before = li > 0 ? c->layers + li - 1 : nullptr;
  StartArgs a{};
  a.x = w->x;
  a.rows = L || all ? nullptr : b->want;
  const int n = L || all ? b->n : b->n_want;
  if (n <= 0) return BB_OK;
  a.embed = li == 0;
  a.tok = b->tok;
  a.pos = b->pos;
  a.emb = c->embed;
  a.pos_tab = c->pos;
  a.emb_scale = c->embed_scale;
  a.vocab = c->vocab;
  a.max_pos = c->max_pos;
  if (before && before->n_experts > 0) {
    a.ex_out = w->ex_out;
    a.pair_row = w->pair_row;
    a.pair_w = w->pair_w;
    a.top = before->top;
  }
  a.w = L ? L->norm : c->final_norm;
  a.bias = L ? L->down_b : nullptr;
  a.write = L && (a.embed || a.top > 0 || a.bias);
  a.d = c->width;
  a.dp = c->dp;
  a.eps = c->eps;
  a.counts = w->ex_count;
  a.n_counts = L ? L->n_experts : 0;
  a.trace = trace;
  cudaStream_t s = (cudaStream_t)stream;
  void* h = L ? w->h : w->hn;
  if (c->dtype) hy_start_kernel<float><<<n, ROW_THREADS, 0, s>>>(a, static_cast<float*>(h));
  else hy_start_kernel<__nv_bfloat16><<<n, ROW_THREADS, 0, s>>>(a, static_cast<__nv_bfloat16*>(h));
  return (int)cudaGetLastError();
}

BB_API int bb_hy_kv_post(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? launch_kv_post<float>(*c, *L, *w, *b, (cudaStream_t)stream)
                  : launch_kv_post<__nv_bfloat16>(*c, *L, *w, *b, (cudaStream_t)stream);
}

BB_API int bb_hy_glu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0 || L->ff <= 0) return BB_OK;
  return c->dtype ? launch_glu<float>(*L, *w, n, (cudaStream_t)stream) : launch_glu<__nv_bfloat16>(*L, *w, n, (cudaStream_t)stream);
}

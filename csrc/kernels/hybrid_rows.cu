// Row kernels of the hybrid decoder, one block per token row, fp32 arithmetic, bf16 or fp32 storage:
//   hy_embed_norm   embedding row -> RMS norm -> fp32 residual stream
//   hy_norm         residual row (optionally picked by an index list) -> RMS norm -> projection input
//   hy_attn_post    after the fused input projection of an attention layer: RMS norm over the whole q and
//                   the whole k, partial rotation, value mixing with an earlier layer, K/V written
//                   straight into the sequence's page, and the layer's gated feed-forward product
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

// Blocks of a "post" launch: blockIdx.y = 0 is the row's mixer part, every further one GLU_COLS columns of
// its feed-forward product (GLU_VECS vectors of a thread, all asked for before the first is used).
constexpr int GLU_VECS = 3;
constexpr int GLU_COLS = ROW_THREADS * 8 * GLU_VECS;

template <typename T>
__device__ __forceinline__ void glu_part(const BbHyLayer& L, const T* row, T* crow) {
  struct alignas(sizeof(T) * 8) Raw {
    T v[8];
  };
  const int n = (L.ff + 7) & ~7, i0 = (blockIdx.y - 1) * GLU_COLS + threadIdx.x * 8;
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
#pragma unroll
      for (int j = 0; j < 8; ++j)
        f[j] = clamped_glu_as<T>(to_f(g[t].v[j]), to_f(u[t].v[j]), L.glu_limit, L.glu_alpha, L.glu_shift);
      store8(crow + L.off_act + i, f);
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
    glu_part(L, row, cat + (size_t)r * ldc);
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
    glu_part(L, row, cat + (size_t)r * ldc);
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

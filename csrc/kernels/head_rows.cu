// Rows of heads between a projection and its mixer, fp32 arithmetic, bf16 or fp32 storage:
//   hy_heads   per head: root-mean-square norm with one gain for all heads, rotation of neighbouring pairs; queries in
//              place, keys and (rotated) values into the sequence's page, or keys in place too where there are no pages.
//              A single token that ends a block of the pooled cache also writes the block's means
//   hy_pool    means of the blocks that end in prompt portions, and the means that their queries see as rows of one
//              matrix for the flash kernel
// A block's mean lies in the page of its last token, at that token's offset / pool: pages hold ceil(block_size / pool)
// of them, the page table is the tokens', and a reused page needs no clearing.
#include "../common/host.hpp"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int HR_THREADS = 256;

// Where the mean of the block that ends at position e lies, in rows of pool_rows per page and head.
struct PoolPlace {
  int blk, off;
};
__device__ __forceinline__ PoolPlace pool_place(const BbHyLayer& L, const int* bt, int e, int bs) {
  return {bt[e / bs], e % bs / L.pool};
}

// Eight channels of the mean of block `blk` (vector v of keys, then values of all heads) from the pages; the pages may
// have been written by this block, so the loads are plain ones.
template <typename T>
__device__ __forceinline__ void pool_vector(const BbHyLayer& L, const int* bt, int bs, int blk, int v, float (&m)[8], bool& key,
                                            int& head, int& col) {
  const int nk = L.hk * L.dkp / 8;
  key = v < nk;
  const int size = key ? L.dkp : L.dvp, i = (key ? v : v - nk) * 8;
  head = i / size;
  col = i - head * size;
  const T* pages = static_cast<const T*>(key ? L.kc : L.vc);
#pragma unroll
  for (int j = 0; j < 8; ++j) m[j] = 0.f;
  const int p0 = blk * L.pool;
#pragma unroll 4
  for (int t = 0; t < L.pool; ++t) {
    const int p = p0 + t;
    float f[8];
    load8(pages + (((size_t)bt[p / bs] * L.hk + head) * bs + p % bs) * size + col, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) m[j] += f[j];
  }
  const float inv = 1.f / (float)L.pool;
#pragma unroll
  for (int j = 0; j < 8; ++j) m[j] *= inv;
}

template <typename T>
__device__ __forceinline__ T* pool_row(const BbHyLayer& L, bool key, PoolPlace at, int head) {
  T* base = static_cast<T*>(key ? L.pkc : L.pvc);
  return base + (((size_t)at.blk * L.hk + head) * L.pool_rows + at.off) * (key ? L.dkp : L.dvp);
}

// (u, v) of neighbouring channels turned by the row's angles; c: channel of f[0].
__device__ __forceinline__ void turn_pairs(float (&f)[8], const float* ct, const float* st, int c, int rot) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int i = (c >> 1) + j;
    if (2 * i < rot) {
      const float co = ct[i], si = st[i], u = f[2 * j], v = f[2 * j + 1];
      f[2 * j] = fmaf(u, co, -v * si);
      f[2 * j + 1] = fmaf(v, co, u * si);
    }
  }
}

// `lanes` threads (a power of two up to a warp) share a head.
template <typename T>
__global__ void __launch_bounds__(HR_THREADS)
hy_heads_kernel(const __grid_constant__ BbHyLayer L, T* proj, int ld, const int* __restrict__ pos_,
                const int* __restrict__ row_seq, const int* __restrict__ tables, int max_blocks, int bs, int n_pre, int hq,
                int hk, int off_k, int lanes, float eps) {
  const int r = blockIdx.x, lane = threadIdx.x % lanes, group = threadIdx.x / lanes, groups = blockDim.x / lanes;
  T* row = proj + (size_t)r * ld;
  const int pos = pos_[r];
  const bool paged = L.kc != nullptr;
  const int* bt = paged ? tables + (size_t)row_seq[r] * max_blocks : nullptr;
  const int blk = paged ? bt[pos / bs] : 0, off = pos % bs;
  const int heads = hq + hk + (paged ? hk : 0);
  for (int h0 = 0; h0 < heads; h0 += groups) {
    const bool live = h0 + group < heads;
    const int u = live ? h0 + group : 0, part = u < hq ? 0 : (u < hq + hk ? 1 : 2);
    const int h = part == 0 ? u : (part == 1 ? u - hq : u - hq - hk);
    const int size = part == 2 ? L.dvp : L.dkp, vecs = size / 8;
    T* src = row + (part == 0 ? L.off_q : (part == 1 ? off_k : L.off_v)) + h * size;
    T* dst = part == 0 || !paged
                 ? src
                 : static_cast<T*>(part == 1 ? L.kc : L.vc) + (((size_t)blk * L.hk + h) * bs + off) * size;
    const float* gain = part == 0 ? L.q_norm : (part == 1 ? L.k_norm : nullptr);
    const float *ct = part == 2 ? L.vcos_t : L.cos_t, *st = part == 2 ? L.vsin_t : L.sin_t;
    const int rot = !ct ? 0 : (part == 2 ? L.dv : L.rot);
    float f[8], ss = 0.f;
    for (int v = lane; live && v < vecs; v += lanes) {
      load8(src + v * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rstd = gain ? 1.f / sqrtf(ss / (float)L.dk + eps) : 1.f;
    for (int v = lane; live && v < vecs; v += lanes) {
      if (vecs > lanes) load8(src + v * 8, f);
      if (gain) {
        float g[8];
        load8(gain + v * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= rstd * g[j];
      }
      if (rot) turn_pairs(f, ct + (size_t)pos * (rot >> 1), st + (size_t)pos * (rot >> 1), v * 8, rot);
      store8(dst + v * 8, f);
    }
  }
  if (r >= n_pre && L.pool && (pos + 1) % L.pool == 0) {
    __syncthreads();
    const PoolPlace at = pool_place(L, bt, pos, bs);
    for (int v = threadIdx.x; v < L.hk * (L.dkp + L.dvp) / 8; v += blockDim.x) {
      float m[8];
      bool key;
      int head, col;
      pool_vector<T>(L, bt, bs, pos / L.pool, v, m, key, head, col);
      store8(pool_row<T>(L, key, at, head) + col, m);
    }
  }
}

// blockIdx.x: block of the sequence blockIdx.y.  seen (may be null): [rows][ld] keys | values of all heads, block b of
// the sequence at row ctx_row0 / pool + b.
template <typename T>
__global__ void __launch_bounds__(HR_THREADS)
hy_pool_kernel(const __grid_constant__ BbHyLayer L, const int* __restrict__ tables, int max_blocks, int bs,
               const int* __restrict__ seq_pos0, const int* __restrict__ seq_ctx, const int* __restrict__ ctx_row0, T* seen,
               int ld) {
  const int s = blockIdx.y, b = blockIdx.x, ctx = seq_ctx[s], end = (b + 1) * L.pool;
  if (end > ctx) return;
  const bool fresh = end > seq_pos0[s], shown = seen && end <= ctx - L.window;
  if (!fresh && !shown) return;
  const int* bt = tables + (size_t)s * max_blocks;
  const PoolPlace at = pool_place(L, bt, end - 1, bs);
  const int nk = L.hk * L.dkp / 8;
  for (int v = threadIdx.x; v < L.hk * (L.dkp + L.dvp) / 8; v += HR_THREADS) {
    float m[8];
    bool key;
    int head, col;
    if (fresh) {
      pool_vector<T>(L, bt, bs, b, v, m, key, head, col);
      store8(pool_row<T>(L, key, at, head) + col, m);
    } else {
      key = v < nk;
      const int size = key ? L.dkp : L.dvp, i = (key ? v : v - nk) * 8;
      head = i / size;
      col = i - head * size;
      load8(pool_row<T>(L, key, at, head) + col, m);
    }
    if (shown) store8(seen + (size_t)(ctx_row0[s] / L.pool + b) * ld + v * 8, m);
  }
}

template <typename T>
static int launch_heads(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, int bs, int rows, int hq, int hk, int off_k,
                        float eps, cudaStream_t s) {
  const int widest = (L.kc && L.dvp > L.dkp ? L.dvp : L.dkp) / 8;
  int lanes = 1;
  while (lanes < widest && lanes < 32) lanes <<= 1;
  int threads = (hq + hk + (L.kc ? hk : 0)) * lanes;
  threads = threads > HR_THREADS ? HR_THREADS : (threads + 31) & ~31;
  hy_heads_kernel<T><<<rows, threads, 0, s>>>(L, static_cast<T*>(w.proj), w.ld_proj, b.pos, b.row_seq, b.tables, b.max_blocks,
                                              bs, b.n_pre, hq, hk, off_k, lanes, eps);
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

// Queries, keys and values of every row of an attention layer.
BB_API int bb_hy_heads(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->n <= 0) return BB_OK;
  if (L->hq % L->hk || L->dkp % 8 || L->dvp % 8 || (L->pool && L->pool_rows * L->pool < c->block_size)) return BB_EARG;
  return c->dtype ? launch_heads<float>(*L, *w, *b, c->block_size, b->n, L->hq, L->hk, L->off_k, c->eps, (cudaStream_t)stream)
                  : launch_heads<__nv_bfloat16>(*L, *w, *b, c->block_size, b->n, L->hq, L->hk, L->off_k, c->eps, (cudaStream_t)stream);
}

// Rotation of the queries and keys of the prompt portions of a linear attention layer, in place.
BB_API int bb_hy_turn(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->n_pre <= 0 || !L->rot) return BB_OK;
  BbHyLayer t = *L;
  t.kc = nullptr;
  t.q_norm = t.k_norm = nullptr;
  t.pool = 0;
  t.dk = L->n;
  t.dkp = L->np;
  return c->dtype ? launch_heads<float>(t, *w, *b, c->block_size, b->n_pre, L->heads, L->heads, L->off_kk, 0.f, (cudaStream_t)stream)
                  : launch_heads<__nv_bfloat16>(t, *w, *b, c->block_size, b->n_pre, L->heads, L->heads, L->off_kk, 0.f,
                                                (cudaStream_t)stream);
}

// Pooled blocks of the prompt portions; `gather`: those that their queries see -> w->pk.
BB_API int bb_hy_pool(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int gather, void* stream) {
  if (b->ns_pre <= 0 || !L->pool || b->max_ctx < L->pool) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const dim3 grid(b->max_ctx / L->pool, b->ns_pre);
#define BB_POOL(T)                                                                                                          \
  hy_pool_kernel<T><<<grid, HR_THREADS, 0, s>>>(*L, b->tables, b->max_blocks, c->block_size, b->seq_pos0, b->seq_ctx, b->ctx_row0, \
                                                gather ? static_cast<T*>(w->pk) : nullptr, w->ld_pk)
  if (c->dtype) BB_POOL(float);
  else BB_POOL(__nv_bfloat16);
#undef BB_POOL
  return (int)cudaGetLastError();
}

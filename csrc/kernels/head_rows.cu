// Rows of heads between a projection and its mixer, fp32 arithmetic, bf16 or fp32 storage:
//   hy_heads, hy_head_rows (portions as a list of heads; a row to a block)
//              per head: root-mean-square norm with one gain for all heads, rotation of neighbouring pairs; queries in
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
#pragma unroll 8
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

// Angles of the four pairs from channel c on (pairs past the rotated part stay where they are).
__device__ __forceinline__ void load_angles(const float* ct, const float* st, int c, int rot, float (&co)[4], float (&si)[4]) {
  const int i = c >> 1;
  if (c + 8 <= rot && (rot & 7) == 0) {
    const float4 a = *reinterpret_cast<const float4*>(ct + i), b = *reinterpret_cast<const float4*>(st + i);
    co[0] = a.x; co[1] = a.y; co[2] = a.z; co[3] = a.w;
    si[0] = b.x; si[1] = b.y; si[2] = b.z; si[3] = b.w;
  } else {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const bool in = 2 * (i + j) < rot;
      co[j] = in ? ct[i + j] : 1.f;
      si[j] = in ? st[i + j] : 0.f;
    }
  }
}
// (u, v) of neighbouring channels turned by them
__device__ __forceinline__ void turn_pairs(float (&f)[8], const float (&co)[4], const float (&si)[4]) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float u = f[2 * j], v = f[2 * j + 1];
    f[2 * j] = fmaf(u, co[j], -v * si[j]);
    f[2 * j + 1] = fmaf(v, co[j], u * si[j]);
  }
}

// A single token that ends a block: the block's means (the row's keys and values are written; every thread comes here).
template <typename T>
__device__ __forceinline__ void pool_single(const BbHyLayer& L, const int* bt, int bs, int pos) {
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

struct HeadArgs {
  const int *pos, *row_seq, *tables;
  int ld, max_blocks, bs, rows, n_pre, hq, hk, off_k, lanes;
  float eps;
};
// A head of a row: queries, then keys, then values.
template <typename T>
struct HeadOf {
  int part, h, size, rot, src;       // src: its first column in the projection
  const float *gain, *ct, *st;
  __device__ HeadOf(const BbHyLayer& L, const HeadArgs& a, int u) {
    part = u < a.hq ? 0 : (u < a.hq + a.hk ? 1 : 2);
    h = part == 0 ? u : (part == 1 ? u - a.hq : u - a.hq - a.hk);
    size = part == 2 ? L.dvp : L.dkp;
    src = (part == 0 ? L.off_q : (part == 1 ? a.off_k : L.off_v)) + h * size;
    gain = part == 0 ? L.q_norm : (part == 1 ? L.k_norm : nullptr);
    ct = part == 2 ? L.vcos_t : L.cos_t;
    st = part == 2 ? L.vsin_t : L.sin_t;
    rot = !ct ? 0 : (part == 2 ? L.dv : L.rot);
  }
  __device__ T* page(const BbHyLayer& L, const HeadArgs& a, int blk, int pos) const {
    return static_cast<T*>(part == 1 ? L.kc : L.vc) + (((size_t)blk * L.hk + h) * a.bs + pos % a.bs) * size;
  }
};

// Rows of prompt portions: `lanes` threads (a power of two up to a warp) share a head of one row and have a vector of it
// each; rows and heads are one list, so that no warp waits for another.
template <typename T>
__global__ void __launch_bounds__(HR_THREADS, sizeof(T) == 2 ? 6 : 4)
hy_heads_kernel(const __grid_constant__ BbHyLayer L, T* proj, const __grid_constant__ HeadArgs a, int heads) {
  const int lane = threadIdx.x % a.lanes, unit = blockIdx.x * (HR_THREADS / a.lanes) + threadIdx.x / a.lanes, r = unit / heads;
  const HeadOf<T> x(L, a, unit - r * heads);
  const bool live = r < a.rows && lane * 8 < x.size;
  T* src = proj + (size_t)r * a.ld + x.src + lane * 8;
  float f[8] = {}, co[4], si[4], ss = 0.f;
  T* dst = src;
  if (live) {
    load8(src, f);
    const int pos = a.pos[r];
    load_angles(x.ct + (size_t)pos * (x.rot >> 1), x.st + (size_t)pos * (x.rot >> 1), lane * 8, x.rot, co, si);
    if (x.part > 0 && L.kc)
      dst = x.page(L, a, a.tables[(size_t)a.row_seq[r] * a.max_blocks + pos / a.bs], pos) + lane * 8;
  }
  if (L.q_norm) {
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    for (int o = 1; o < a.lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  }
  if (!live) return;
  if (x.gain) {
    float g[8];
    load8(x.gain + lane * 8, g);
    const float rstd = 1.f / sqrtf(ss / (float)L.dk + a.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= rstd * g[j];
  }
  turn_pairs(f, co, si);
  store8(dst, f);
}

// The same with a row to a block: single tokens, and heads wider than a warp has vectors for.
template <typename T>
__global__ void __launch_bounds__(HR_THREADS)
hy_head_rows_kernel(const __grid_constant__ BbHyLayer L, T* proj, const __grid_constant__ HeadArgs a, int r0) {
  const int r = r0 + blockIdx.x, lane = threadIdx.x % a.lanes, group = threadIdx.x / a.lanes, groups = blockDim.x / a.lanes;
  const bool paged = L.kc != nullptr;
  const int pos = a.pos[r], heads = a.hq + a.hk + (paged ? a.hk : 0);
  const int* bt = paged ? a.tables + (size_t)a.row_seq[r] * a.max_blocks : nullptr;
  for (int h0 = 0; h0 < heads; h0 += groups) {
    const bool live = h0 + group < heads;
    const HeadOf<T> x(L, a, live ? h0 + group : 0);
    const int vecs = x.size / 8;
    T* src = proj + (size_t)r * a.ld + x.src;
    T* dst = x.part > 0 && paged ? x.page(L, a, bt[pos / a.bs], pos) : src;
    float f[8], ss = 0.f;
    for (int v = lane; live && v < vecs; v += a.lanes) {
      load8(src + v * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    for (int o = 1; o < a.lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rstd = x.gain ? 1.f / sqrtf(ss / (float)L.dk + a.eps) : 1.f;
    for (int v = lane; live && v < vecs; v += a.lanes) {
      float g[8], co[4], si[4];
      load8(src + v * 8, f);
      if (x.gain) {
        load8(x.gain + v * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= rstd * g[j];
      }
      load_angles(x.ct + (size_t)pos * (x.rot >> 1), x.st + (size_t)pos * (x.rot >> 1), v * 8, x.rot, co, si);
      turn_pairs(f, co, si);
      store8(dst + v * 8, f);
    }
  }
  if (r >= a.n_pre && L.pool && (pos + 1) % L.pool == 0) pool_single<T>(L, bt, a.bs, pos);
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
  const int widest = (L.kc && L.dvp > L.dkp ? L.dvp : L.dkp) / 8, heads = hq + hk + (L.kc ? hk : 0);
  int lanes = 1;
  while (lanes < widest && lanes < 32) lanes <<= 1;
  const int listed = widest <= lanes ? b.n_pre : 0;      // rows that go as a list of heads
  const HeadArgs a{b.pos, b.row_seq, b.tables, w.ld_proj, b.max_blocks, bs, listed, b.n_pre, hq, hk, off_k, lanes, eps};
  T* proj = static_cast<T*>(w.proj);
  if (listed > 0)
    hy_heads_kernel<T><<<(int)(((long)listed * heads * lanes + HR_THREADS - 1) / HR_THREADS), HR_THREADS, 0, s>>>(L, proj, a, heads);
  if (rows > listed) {
    const int threads = heads * lanes < HR_THREADS ? (heads * lanes + 31) & ~31 : HR_THREADS;
    hy_head_rows_kernel<T><<<rows - listed, threads, 0, s>>>(L, proj, a, listed);
  }
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

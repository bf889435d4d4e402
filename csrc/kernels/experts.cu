// Mixture of experts of a serving step, everything but its matrix products, for bf16 and fp32 storage:
//   hy_route         one warp per token: softmax over the router's fp32 logits, the best groups by their best
//                    expert, the best experts of those, their weights; a place among the rows of each
//   hy_products, hy_route_row   few rows: the router's products by slices of channels, added up where a block per row
//                    routes
//   hy_expert_rows   rows of the normed input to their experts' places, every expert's rows on 128-row tiles of
//                    their own; the tiles' experts
//   hy_expert_glu    clamped gated product of the experts' two halves
// A row's place inside its expert's tiles depends on the order in which blocks arrive; its values do not.  The
// weighted sum over a token's experts is taken where the next layer starts (hy_start).
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int EX_THREADS = 256;

// Largest value of the warp and the lowest index that has it, in every lane.
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
    const int i2 = __shfl_xor_sync(0xffffffffu, i, o);
    if (v2 > v || (v2 == v && i2 < i)) {
      v = v2;
      i = i2;
    }
  }
}

// The choices of one token by one warp: lane c < top gets the c-th expert and its weight.  V: experts of a lane
// (expert j * 32 + lane).  Scores are a softmax, the weights over the chosen ones' sum, or the sigmoid of every logit as it is.
template <int V>
__device__ __forceinline__ void choose(const BbHyLayer& L, const float* logits, int& my_e, float& my_w) {
  const int lane = threadIdx.x & 31, E = L.n_experts, size = E / L.groups_all;
  float s[V], mx = -INFINITY, sum = 0.f;
#pragma unroll
  for (int j = 0; j < V; ++j) {
    s[j] = j * 32 + lane < E ? logits[j * 32 + lane] : -INFINITY;
    mx = fmaxf(mx, s[j]);
  }
  if (L.score_kind == 0) {
    mx = warp_max(mx);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      s[j] = j * 32 + lane < E ? expf(s[j] - mx) : 0.f;
      sum += s[j];
    }
    const float inv = 1.f / warp_sum(sum);
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] *= inv;
  } else {
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = sigmoid_f(s[j]);
  }
  // groups: take the best expert left in any group not yet kept, keep its group
  bool kept[V];
#pragma unroll
  for (int j = 0; j < V; ++j) kept[j] = L.groups_keep >= L.groups_all;
  auto best_of = [&](bool in, int& bi) {
    float best = -1.f;
    bi = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const int e = j * 32 + lane;
      if (e < E && kept[j] == in && s[j] > best) {
        best = s[j];
        bi = e;
      }
    }
    warp_best(best, bi);
    return best;
  };
  if (L.groups_keep < L.groups_all)
    for (int g = 0; g < L.groups_keep; ++g) {
      int bi;
      best_of(false, bi);
      const int first = bi / size * size;
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const int e = j * 32 + lane;
        if (e >= first && e < first + size) kept[j] = true;
      }
    }
  float total = 0.f;
  my_w = 0.f;
  my_e = 0;
  for (int c = 0; c < L.top; ++c) {
    int bi;
    const float best = best_of(true, bi);
#pragma unroll
    for (int j = 0; j < V; ++j)
      if (j * 32 + lane == bi) kept[j] = false;
    total += best;
    if (lane == c) {
      my_w = best;
      my_e = min(bi, E - 1);                       // (logits that are not numbers pick no expert)
    }
  }
  my_w = (L.score_kind == 0 ? my_w / (total + L.route_tiny) : my_w) * L.route_scale;
}

template <int V>
__global__ void __launch_bounds__(EX_THREADS)
hy_route_kernel(const __grid_constant__ BbHyLayer L, const float* __restrict__ logits, int ld, int* __restrict__ pair_expert,
                int* __restrict__ pair_row, float* __restrict__ pair_w, int* __restrict__ count, int n) {
  __shared__ int hist[V * 32];
  const int lane = threadIdx.x & 31, E = L.n_experts, t = blockIdx.x * (EX_THREADS / 32) + (threadIdx.x >> 5);
  for (int e = threadIdx.x; e < E; e += EX_THREADS) hist[e] = 0;
  __syncthreads();
  const bool mine = t < n && lane < L.top;
  const size_t p = (size_t)t * L.top + lane;
  int e = 0, place = 0;
  if (t < n) {
    float w;
    choose<V>(L, logits + (size_t)t * ld, e, w);
    if (mine) {
      pair_expert[p] = e;
      pair_w[p] = w;
      place = atomicAdd(&hist[e], 1);              // place among the block's rows of this expert
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < E; i += EX_THREADS)
    if (hist[i] > 0) hist[i] = atomicAdd(&count[i], hist[i]);   // ... and the block's first place among all
  __syncthreads();
  if (mine) pair_row[p] = hist[e] + place;
}

// Few rows: the fp32 products of the normed input (router logits, gates) by slices of PR_K channels side by side, ...
constexpr int PR_TILE = 64, PR_K = 64;

template <typename T>
__global__ void __launch_bounds__(EX_THREADS)
hy_products_kernel(const T* __restrict__ h, const T* __restrict__ W, int dp, int n, int n_out, float* __restrict__ part) {
  __shared__ float sa[PR_TILE][PR_K + 1], sb[PR_TILE][PR_K + 1];
  const int k0 = blockIdx.x * PR_K, o0 = blockIdx.y * PR_TILE, r0 = blockIdx.z * PR_TILE;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  struct alignas(sizeof(T) * 8) Raw {
    T v[8];
  };
  constexpr int IT = PR_TILE * PR_K / 8 / EX_THREADS;
  Raw a[IT], b[IT];
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int v = threadIdx.x + i * EX_THREADS, r = v / (PR_K / 8), k = k0 + v % (PR_K / 8) * 8;
    if (r0 + r < n && k < dp) a[i] = *reinterpret_cast<const Raw*>(h + (size_t)(r0 + r) * dp + k);
    if (o0 + r < n_out && k < dp) b[i] = *reinterpret_cast<const Raw*>(W + (size_t)(o0 + r) * dp + k);
  }
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int v = threadIdx.x + i * EX_THREADS, r = v / (PR_K / 8), c = v % (PR_K / 8) * 8;
    const bool in = k0 + c < dp;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      sa[r][c + j] = in && r0 + r < n ? to_f(a[i].v[j]) : 0.f;
      sb[r][c + j] = in && o0 + r < n_out ? to_f(b[i].v[j]) : 0.f;
    }
  }
  __syncthreads();
  float acc[4][4] = {};
#pragma unroll 8
  for (int k = 0; k < PR_K; ++k) {
    float x[4], w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[i] = sa[ty + 16 * i][k];
      w[i] = sb[tx + 16 * i][k];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = r0 + ty + 16 * i, o = o0 + tx + 16 * j;
      if (r < n && o < n_out) part[((size_t)blockIdx.x * n + r) * n_out + o] = acc[i][j];
    }
}

// ... then one block per row adds the slices up, in order, and routes.  V = 0: nothing to route.
template <int V>
__global__ void __launch_bounds__(EX_THREADS)
hy_route_row_kernel(const __grid_constant__ BbHyLayer L, const float* __restrict__ part, int slices,
                    float* __restrict__ out, int ld, int* __restrict__ pair_expert, int* __restrict__ pair_row,
                    float* __restrict__ pair_w, int* __restrict__ count) {
  extern __shared__ float s_out[];                 // [n_out], then [threads / n_out][n_out]
  const int r = blockIdx.x, n = gridDim.x, n_out = L.in32.n, lane = threadIdx.x & 31;
  const int per = max(EX_THREADS / n_out, 1);      // threads of an output
  for (int o = threadIdx.x % n_out, g = threadIdx.x / n_out; o < n_out && g < per; o += EX_THREADS) {
    float a = 0.f;
    const int s0 = slices * g / per, s1 = slices * (g + 1) / per;
#pragma unroll 8
    for (int s = s0; s < s1; ++s) a += part[((size_t)s * n + r) * n_out + o];
    s_out[n_out * (1 + g) + o] = a;
  }
  __syncthreads();
  for (int o = threadIdx.x; o < n_out; o += EX_THREADS) {
    float a = 0.f;
    for (int g = 0; g < per; ++g) a += s_out[n_out * (1 + g) + o];
    s_out[o] = a;
    out[(size_t)r * ld + o] = a;
  }
  if constexpr (V > 0) {
    __syncthreads();
    if (threadIdx.x < 32) {
      int e;
      float w;
      choose<V>(L, s_out, e, w);
      if (lane < L.top) {
        const size_t p = (size_t)r * L.top + lane;
        pair_expert[p] = e;
        pair_w[p] = w;
        pair_row[p] = atomicAdd(&count[e], 1);
      }
    }
  }
}

// Every expert's first row, from the counts: rows of expert e start on a 128-row tile.
__device__ __forceinline__ void expert_offsets(const int* count, int E, int* off) {
  if (threadIdx.x < 32) {
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x, c = e < E ? (count[e] + 127) & ~127 : 0;
      int x = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if ((int)threadIdx.x >= o) x += y;
      }
      if (e < E) off[e] = base + x - c;
      base += __shfl_sync(0xffffffffu, x, 31);
    }
    if (threadIdx.x == 0) off[E] = base;
  }
  __syncthreads();
}

// A warp per token (its row times the expert's weight, where that multiplies the input); the last block writes every tile's expert and, cap entries further, how many rows it has.
template <typename T>
__global__ void __launch_bounds__(EX_THREADS)
hy_expert_rows_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ h, int dp, const int* __restrict__ pair_expert,
                      int* __restrict__ pair_row, const float* __restrict__ pair_w, const int* __restrict__ count,
                      T* __restrict__ out, int* __restrict__ tiles, int n_tiles, int cap, int n) {
  extern __shared__ int off[];
  const int E = L.n_experts;
  expert_offsets(count, E, off);
  if (blockIdx.x == gridDim.x - 1) {
    for (int t = threadIdx.x; t < n_tiles; t += EX_THREADS) {
      int e = -1;
      if (t * 128 < off[E]) {
        int lo = 0, hi = E - 1;                   // the last expert that starts at or before the tile
        while (lo < hi) {
          const int mid = (lo + hi + 1) >> 1;
          if (off[mid] <= t * 128) lo = mid; else hi = mid - 1;
        }
        e = lo;
      }
      tiles[t] = e;
      tiles[cap + t] = e < 0 ? 0 : min(count[e] - (t * 128 - off[e]), 128);
    }
    return;
  }
  const int lane = threadIdx.x & 31, t = blockIdx.x * (EX_THREADS / 32) + (threadIdx.x >> 5);
  if (t >= n) return;
  int row = 0;
  float weight = 1.f;
  if (lane < L.top) {
    const size_t p = (size_t)t * L.top + lane;
    if (L.weigh_input) weight = pair_w[p];
    row = min(off[pair_expert[p]] + pair_row[p], n_tiles * 128 - 1);
    pair_row[p] = row;
  }
  struct alignas(16) Vec {
    T v[16 / sizeof(T)];
  };
  constexpr int VN = 16 / sizeof(T);
  const Vec* src = reinterpret_cast<const Vec*>(h + (size_t)t * dp);
  constexpr int U = 4;
  for (int i0 = 0; i0 < dp / VN; i0 += 32 * U) {
    Vec x[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u * 32 + lane < dp / VN) x[u] = src[i0 + u * 32 + lane];
    for (int c = 0; c < L.top; ++c) {
      Vec* dst = reinterpret_cast<Vec*>(out + (size_t)__shfl_sync(0xffffffffu, row, c) * dp);
      const float w = __shfl_sync(0xffffffffu, weight, c);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (i0 + u * 32 + lane >= dp / VN) continue;
        Vec y = x[u];
        if (L.weigh_input) {
#pragma unroll
          for (int j = 0; j < VN; ++j) y.v[j] = from_f<T>(to_f(y.v[j]) * w);
        }
        dst[i0 + u * 32 + lane] = y;
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(EX_THREADS)
hy_expert_glu_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ gu, int ldgu, T* __restrict__ act, int lda,
                     const int* __restrict__ tile_rows, int tile_blocks) {
  const int tile = blockIdx.x / tile_blocks;
  const int vecs = L.effp / 8, total = tile_rows[tile] * vecs, stride = tile_blocks * EX_THREADS;
  for (int i = (blockIdx.x % tile_blocks) * EX_THREADS + threadIdx.x; i < total; i += stride) {
    const size_t r = (size_t)tile * 128 + i / vecs;
    const int c = i % vecs * 8;
    float g[8], u[8];
    load8(gu + r * ldgu + c, g);
    load8(gu + r * ldgu + L.effp + c, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] = clamped_glu_as<T>(g[j], u[j], L.e_limit, L.e_alpha, L.e_shift);
    store8(act + r * lda + c, g);
  }
}

}  // namespace bb

using namespace bb;

// Tiles that n tokens of the layer can take.
static int moe_tiles(const BbHyLayer& L, int n) {
  const long pairs = (long)n * L.top;
  return (int)(pairs / 128 + (pairs < L.n_experts ? pairs : L.n_experts));
}
BB_API int bb_hy_moe_tiles(const BbHyLayer* L, int n) { return moe_tiles(*L, n); }

// Router logits in columns [0, experts) of w->f32; the counts are clear (hy_start).
BB_API int bb_hy_route(const BbHyCfg*, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  const int E = L->n_experts;
  if (E > 1024 || L->top > 32) return BB_ESIZE;
  cudaStream_t s = (cudaStream_t)stream;
  const int grid = (n + EX_THREADS / 32 - 1) / (EX_THREADS / 32);
#define BB_ROUTE(V) \
  hy_route_kernel<V><<<grid, EX_THREADS, 0, s>>>(*L, w->f32, w->ld_f32, w->pair_expert, w->pair_row, w->pair_w, w->ex_count, n)
  if (E <= 32) BB_ROUTE(1);
  else if (E <= 64) BB_ROUTE(2);
  else if (E <= 128) BB_ROUTE(4);
  else if (E <= 256) BB_ROUTE(8);
  else BB_ROUTE(32);
#undef BB_ROUTE
  return (int)cudaGetLastError();
}

// The fp32 products of the normed input -> w->f32, and with experts the routing; for few rows.  BB_ESIZE for more rows
// than w->part32 holds slices of, and for sizes it does not cover.
BB_API int bb_hy_route_row(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  const int E = L->n_experts, n_out = L->in32.n, slices = (c->dp + PR_K - 1) / PR_K;
  const size_t smem = 4 * (size_t)n_out * (1 + (n_out >= EX_THREADS ? 1 : EX_THREADS / n_out));
  if ((long)slices * n * n_out > w->part32_floats || smem > 48 * 1024 || E > 256 || L->top > 32) return BB_ESIZE;
  cudaStream_t s = (cudaStream_t)stream;
  const dim3 grid(slices, (n_out + PR_TILE - 1) / PR_TILE, (n + PR_TILE - 1) / PR_TILE);
#define BB_PRODUCTS(T)                                                                                       \
  hy_products_kernel<T><<<grid, EX_THREADS, 0, s>>>(static_cast<const T*>(w->h), static_cast<const T*>(L->in32.w), \
                                                    c->dp, n, n_out, w->part32)
  if (c->dtype) BB_PRODUCTS(float);
  else BB_PRODUCTS(__nv_bfloat16);
#undef BB_PRODUCTS
#define BB_ROUTE_ROW(V)                                                                                                        \
  hy_route_row_kernel<V><<<n, EX_THREADS, smem, s>>>(*L, w->part32, slices, w->f32, w->ld_f32, w->pair_expert, w->pair_row, \
                                                     w->pair_w, w->ex_count)
  if (E == 0) BB_ROUTE_ROW(0);
  else if (E <= 32) BB_ROUTE_ROW(1);
  else if (E <= 64) BB_ROUTE_ROW(2);
  else if (E <= 128) BB_ROUTE_ROW(4);
  else BB_ROUTE_ROW(8);
#undef BB_ROUTE_ROW
  return (int)cudaGetLastError();
}

BB_API int bb_hy_expert_rows(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const int tiles = moe_tiles(*L, n), grid = (n + EX_THREADS / 32 - 1) / (EX_THREADS / 32) + 1;
  if (tiles * 128 > w->moe_rows) return BB_EARG;
  const size_t smem = 4 * (size_t)(L->n_experts + 1);
#define BB_ROWS(T)                                                                                           \
  hy_expert_rows_kernel<T><<<grid, EX_THREADS, smem, s>>>(*L, static_cast<const T*>(w->h), c->dp, w->pair_expert, \
                                                          w->pair_row, w->pair_w, w->ex_count, static_cast<T*>(w->ex_in), \
                                                          w->ex_tile, tiles, w->moe_rows / 128, n)
  if (c->dtype) BB_ROWS(float);
  else BB_ROWS(__nv_bfloat16);
#undef BB_ROWS
  return (int)cudaGetLastError();
}

BB_API int bb_hy_expert_glu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const int* rows = w->ex_tile + w->moe_rows / 128;
  const int tiles = moe_tiles(*L, n), per = (128 * (L->effp / 8) + 4 * EX_THREADS - 1) / (4 * EX_THREADS);
#define BB_GLU(T)                                                                                            \
  hy_expert_glu_kernel<T><<<tiles * per, EX_THREADS, 0, s>>>(*L, static_cast<const T*>(w->ex_gu), w->ld_gu,  \
                                                             static_cast<T*>(w->ex_act), w->ld_act, rows, per)
  if (c->dtype) BB_GLU(float);
  else BB_GLU(__nv_bfloat16);
#undef BB_GLU
  return (int)cudaGetLastError();
}

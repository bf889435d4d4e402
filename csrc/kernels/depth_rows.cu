// Row kernels of decoders that pass weighted sums of all layer results on, one block per token row, fp32
// arithmetic:
//   hy_mix_norm    (embedding row, or the weighted sum of the results so far) -> what the next layer adds to
//                  (its feed-forward's output bias included) and its one or two normed inputs
//   hy_polynorm    a N(z) + b N(z^2) + c N(z^3) + e over a row of the up projection, N dividing by the root
//                  mean square -> the feed-forward's part of the row the output projection multiplies
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int MIX_THREADS = 256;

struct MixArgs {
  float* hist;              // results [level][rows, dp]
  size_t level;             // elements between levels
  int levels;               // results that exist (0: the row comes from the embedding)
  const float* weights;     // [levels] (null: the last result alone)
  const int *tok, *rows;    // token ids (levels = 0); row picks (null: in order)
  const void* embed;
  int vocab, d, dp;
  float eps;
  const float *w1, *w2;     // gains of the normed outputs (w2 null: one output)
  void *h1, *h2;
  const float* bias;        // added to the start of the next level (may be null)
  float* trace;             // copy of the row before bias (may be null)
  int start;                // 1: the next level starts from this row
};

// One row at a time per block; rows up to KEEP * 8 * threads wide stay in registers.
template <typename T>
__global__ void __launch_bounds__(MIX_THREADS)
hy_mix_norm_kernel(const __grid_constant__ MixArgs a) {
  __shared__ float buf[32];
  const int out_row = blockIdx.x, r = a.rows ? a.rows[out_row] : out_row;
  float* x0 = a.hist + (size_t)r * a.dp;
  const T* e = nullptr;
  if (a.levels == 0) {
    int id = a.tok[r];
    id = id < 0 ? 0 : (id >= a.vocab ? a.vocab - 1 : id);
    e = static_cast<const T*>(a.embed) + (size_t)id * a.dp;
  }
  auto value = [&](int i, float (&f)[8]) {
    if (a.levels == 0) {
      load8(e + i, f);
    } else if (!a.weights) {
      load8(x0 + (size_t)(a.levels - 1) * a.level + i, f);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = 0.f;
#pragma unroll 4
      for (int l = 0; l < a.levels; ++l) {
        float g[8];
        load8(x0 + (size_t)l * a.level + i, g);
        const float w = a.weights[l];
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = fmaf(w, g[j], f[j]);
      }
    }
  };
  constexpr int KEEP = 2;
  const int step = blockDim.x * 8;
  float v[KEEP][8];
  float ss = 0.f;
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = threadIdx.x * 8 + t * step;
    if (i < a.dp) {
      value(i, v[t]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[t][j] * v[t][j];
    }
  }
  for (int i = threadIdx.x * 8 + KEEP * step; i < a.dp; i += step) {
    float f[8];
    value(i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
  }
  ss = block_sum(ss, buf);
  const float rstd = 1.f / sqrtf(ss / (float)a.d + a.eps);
  T* h1 = static_cast<T*>(a.h1) + (size_t)out_row * a.dp;
  T* h2 = static_cast<T*>(a.h2) + (size_t)out_row * a.dp;
  auto emit = [&](int i, float (&f)[8]) {
    if (a.levels == 0 && a.start) store8(x0 + i, f);
    if (a.trace) store8(a.trace + (size_t)r * a.dp + i, f);
    float g[8];
    if (a.start) {
      if (a.bias) {
        load8(a.bias + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) g[j] += f[j];
        store8(x0 + (size_t)max(a.levels, 1) * a.level + i, g);
      } else {
        store8(x0 + (size_t)max(a.levels, 1) * a.level + i, f);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= rstd;
    if (a.w2) {
      load8(a.w2 + i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] *= f[j];
      store8(h2 + i, g);
    }
    load8(a.w1 + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] *= f[j];
    store8(h1 + i, g);
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = threadIdx.x * 8 + t * step;
    if (i < a.dp) emit(i, v[t]);
  }
  for (int i = threadIdx.x * 8 + KEEP * step; i < a.dp; i += step) {
    float f[8];
    value(i, f);
    emit(i, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(MIX_THREADS)
hy_polynorm_kernel(const T* __restrict__ proj, int ld, int off_up, const float* __restrict__ up_b,
                   const float* __restrict__ poly, T* __restrict__ cat, int ldc, int off_act, int ff, float eps) {
  __shared__ float buf[3][32];
  const int n = (ff + 7) & ~7;
  const T* z = proj + (size_t)blockIdx.x * ld + off_up;
  T* out = cat + (size_t)blockIdx.x * ldc + off_act;
  auto value = [&](int i, float (&f)[8]) {
    float b[8];
    load8(z + i, f);
    load8(up_b + i, b);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] += b[j];      // zero in the padding
  };
  constexpr int KEEP = 3;
  const int step = blockDim.x * 8;
  float v[KEEP][8];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](const float (&f)[8]) {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float q = f[j] * f[j], q2 = q * q;
      s2 += q;
      s4 += q2;
      s6 = fmaf(q2, q, s6);
    }
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = threadIdx.x * 8 + t * step;
    if (i < n) {
      value(i, v[t]);
      add(v[t]);
    }
  }
  for (int i = threadIdx.x * 8 + KEEP * step; i < n; i += step) {
    float f[8];
    value(i, f);
    add(f);
  }
  s2 = warp_sum(s2);
  s4 = warp_sum(s4);
  s6 = warp_sum(s6);
  if ((threadIdx.x & 31) == 0) {
    buf[0][threadIdx.x >> 5] = s2;
    buf[1][threadIdx.x >> 5] = s4;
    buf[2][threadIdx.x >> 5] = s6;
  }
  __syncthreads();
  s2 = s4 = s6 = 0.f;
  for (int i = 0; i < (int)blockDim.x >> 5; ++i) {
    s2 += buf[0][i];
    s4 += buf[1][i];
    s6 += buf[2][i];
  }
  const float inv = 1.f / (float)ff;
  const float ca = poly[0] / sqrtf(s2 * inv + eps), cb = poly[1] / sqrtf(s4 * inv + eps);
  const float cc = poly[2] / sqrtf(s6 * inv + eps), ce = poly[3];
  auto emit = [&](int i, float (&f)[8]) {
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = fmaf(f[j], fmaf(f[j], fmaf(f[j], cc, cb), ca), ce);
    store8(out + i, f);
  };
#pragma unroll
  for (int t = 0; t < KEEP; ++t) {
    const int i = threadIdx.x * 8 + t * step;
    if (i < n) emit(i, v[t]);
  }
  for (int i = threadIdx.x * 8 + KEEP * step; i < n; i += step) {
    float f[8];
    value(i, f);
    emit(i, f);
  }
}

static int row_threads(int n) {
  const int t = ((n + 7) / 8 + 31) & ~31;
  return t < 32 ? 32 : (t > MIX_THREADS ? MIX_THREADS : t);
}

}  // namespace bb

using namespace bb;

// Row r of the step before layer `li` (li = n_layers: before the output norm, for the rows in b->want):
// the weighted sum of results 0 .. li (the embedding row for li = 0) -> normed inputs, and the start of
// result li + 1.  `trace` (may be null): fp32 [n][dp] copy of the sum.
BB_API int bb_hy_mix_norm(const BbHyCfg* c, int li, const BbHyWork* w, const BbHyBatch* b, float* trace, void* stream) {
  MixArgs a{};
  const bool last = li == c->n_layers;
  const int n = last ? b->n_want : b->n;
  if (n <= 0) return BB_OK;
  a.hist = w->x;
  a.level = (size_t)w->rows * c->dp;
  a.levels = li == 0 ? 0 : li + 1;
  a.weights = li == 0 ? nullptr : c->layers[li - 1].dwa;
  a.tok = b->tok;
  a.rows = last ? b->want : nullptr;
  a.embed = c->embed;
  a.vocab = c->vocab;
  a.d = c->width;
  a.dp = c->dp;
  a.eps = c->eps;
  a.w1 = last ? c->final_norm : c->layers[li].norm;
  a.w2 = last ? nullptr : c->layers[li].norm2;
  a.h1 = last ? w->hn : w->h;
  a.h2 = w->h2;
  a.bias = last ? nullptr : c->layers[li].down_b;
  a.trace = trace;
  a.start = !last;
  const int t = row_threads(c->dp);
  if (c->dtype) hy_mix_norm_kernel<float><<<n, t, 0, (cudaStream_t)stream>>>(a);
  else hy_mix_norm_kernel<__nv_bfloat16><<<n, t, 0, (cudaStream_t)stream>>>(a);
  return (int)cudaGetLastError();
}

BB_API int bb_hy_polynorm(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0 || L->ff <= 0) return BB_OK;
  const int t = row_threads(L->ff);
  cudaStream_t s = (cudaStream_t)stream;
  if (c->dtype)
    hy_polynorm_kernel<float><<<n, t, 0, s>>>(static_cast<const float*>(w->proj), w->ld_proj, L->off_up, L->up_b, L->poly,
                                              static_cast<float*>(w->cat), w->ld_cat, L->off_act, L->ff, c->eps);
  else
    hy_polynorm_kernel<__nv_bfloat16><<<n, t, 0, s>>>(
        static_cast<const __nv_bfloat16*>(w->proj), w->ld_proj, L->off_up, L->up_b, L->poly,
        static_cast<__nv_bfloat16*>(w->cat), w->ld_cat, L->off_act, L->ff, c->eps);
  return (int)cudaGetLastError();
}

// Row kernels of decoders with several residual streams, fp32 arithmetic, bf16 or fp32 activations:
//   hy_streams   between two sublayers: the result of the one before (a projection, two normed projections side by
//                side, a token's experts, or the embedding) goes into the streams, x_t <- sum_s mix[s, t] x_s + out[t] y,
//                and the next one's input is the layer norm of sum_s in[s] x_s.  One pass over the streams.  Single tokens
//                are also shifted towards the token before them, which their slot holds
//   hy_shift     the same shift for the rows of prompt portions; the slot gets the portion's last input
//   hy_gelu      gelu of a feed-forward's up projection (fp32)
//   hy_cap       logits <- cap tanh(logits / cap)
#include "../common/host.hpp"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int ST_THREADS = 256;

struct StreamArgs {
  float* x;                        // [rows][s][dp]
  const int* rows;                 // row of every block (null: its own)
  const int* tok;
  const void* emb;                 // not null: the streams start from the embedding
  float emb_scale;
  int vocab;
  const void *ya, *yb;             // results; yb not null: both normed, times their gains
  int y32;                         // results are fp32
  float *zero_a, *zero_b;          // rows that the next results are added into (null: none)
  const float *gain_a, *gain_b;
  const void* ex_out;              // a token's experts (top = 0: none)
  const int* pair_row;
  const float* pair_w;             // null: summed as they are
  int top;
  const float *from, *to;          // connections of the sublayer before, and of the next (null: the sum of the streams)
  const float *w, *b;              // gain and bias of the norm
  int s, write, d, dp;
  float eps;
  int *counts, n_counts;           // expert counts that block 0 clears
  float* trace;                    // sum of the streams (null: none)
  // token shift (null: none)
  const float* shift;
  void *state, *before;            // last inputs [slots][dp]; rows below n_pre leave theirs in `before`
  const int *row_seq, *slot, *pos;
  int n_pre;
};

__device__ __forceinline__ float round_as(float v, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float round_as(float v, const float*) { return v; }

// S: the most streams (missing ones have coefficients of zero)
template <typename T, int S>
__global__ void __launch_bounds__(ST_THREADS)
hy_streams_kernel(const __grid_constant__ StreamArgs a, T* __restrict__ h) {
  extern __shared__ __align__(16) float u_row[];
  __shared__ float buf[4][32];
  __shared__ float s_mix[S * S], s_out[S], s_in[S];
  const int r = a.rows ? a.rows[blockIdx.x] : (int)blockIdx.x, step = blockDim.x * 8;
  float* xr = a.x + (size_t)r * a.s * a.dp;
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e < a.n_counts; e += blockDim.x) a.counts[e] = 0;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {
    const int s = i / S, t = i % S;
    const bool in = s < a.s && t < a.s;
    s_mix[i] = in && a.from ? a.from[2 * a.s + s * a.s + t] : 0.f;
    if (i < S) {
      s_out[i] = i < a.s && a.from ? a.from[a.s + i] : 0.f;
      s_in[i] = i < a.s ? (a.to ? a.to[i] : 1.f) : 0.f;
    }
  }
  auto result = [&](const void* y, int i, float (&f)[8]) {
    if (sizeof(T) == 2 && a.y32) load8(static_cast<const float*>(y) + (size_t)r * a.dp + i, f);
    else load8(static_cast<const T*>(y) + (size_t)r * a.dp + i, f);
  };
  float fa = 0.f, fb = 0.f;
  if (a.yb) {
    float ssa = 0.f, ssb = 0.f;
    for (int i = threadIdx.x * 8; i < a.dp; i += step) {
      float f[8], g[8];
      result(a.ya, i, f);
      result(a.yb, i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        ssa = fmaf(f[j], f[j], ssa);
        ssb = fmaf(g[j], g[j], ssb);
      }
    }
    ssa = block_sum(ssa, buf[0]);
    ssb = block_sum(ssb, buf[1]);
    fa = 1.f / sqrtf(ssa / (float)a.d + a.eps);
    fb = 1.f / sqrtf(ssb / (float)a.d + a.eps);
  } else {
    __syncthreads();
  }
  const T* er = a.emb ? static_cast<const T*>(a.emb) + (size_t)min(max(a.tok[r], 0), a.vocab - 1) * a.dp : nullptr;
  const int* prow = a.pair_row + (size_t)r * a.top;
  const float* pw = a.pair_w + (size_t)r * a.top;
  float sum = 0.f;
  for (int i = threadIdx.x * 8; i < a.dp; i += step) {
    float u[8] = {}, all[8] = {};
    if (er) {
      float f[8];
      load8(er + i, f);
      float in = 0.f;
#pragma unroll
      for (int t = 0; t < S; ++t) in += s_in[t];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        f[j] *= a.emb_scale;
        u[j] = in * f[j];
      }
#pragma unroll
      for (int t = 0; t < S; ++t)
        if (t < a.s) store8(xr + (size_t)t * a.dp + i, f);
    } else {
      float x[S][8], y[8] = {};
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s < a.s) {
          load8(xr + (size_t)s * a.dp + i, x[s]);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) x[s][j] = 0.f;
        }
      }
      if (a.yb) {
        float f[8], g[8], ga[8], gb[8];
        result(a.ya, i, f);
        result(a.yb, i, g);
        load8(a.gain_a + i, ga);
        load8(a.gain_b + i, gb);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] = fmaf(f[j] * fa, ga[j], g[j] * fb * gb[j]);
      } else if (a.top > 0) {
#pragma unroll 4
        for (int c = 0; c < a.top; ++c) {
          float g[8];
          load8(static_cast<const T*>(a.ex_out) + (size_t)prow[c] * a.dp + i, g);
          const float w = a.pair_w ? pw[c] : 1.f;
#pragma unroll
          for (int j = 0; j < 8; ++j) y[j] = fmaf(w, g[j], y[j]);
        }
      } else {
        result(a.ya, i, y);
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float f[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = s_out[t] * y[j];
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float m = s_mix[s * S + t];
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = fmaf(m, x[s][j], f[j]);
        }
        const float in = s_in[t];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          u[j] = fmaf(in, f[j], u[j]);
          all[j] += f[j];
        }
        if (a.write && t < a.s) store8(xr + (size_t)t * a.dp + i, f);
      }
      if (a.trace) store8(a.trace + (size_t)r * a.dp + i, all);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) sum += u[j];
    store8(u_row + i, u);
    const float none[8] = {};
    if (a.zero_a) store8(a.zero_a + (size_t)r * a.dp + i, none);
    if (a.zero_b) store8(a.zero_b + (size_t)r * a.dp + i, none);
  }
  const float mean = block_sum(sum, buf[2]) / (float)a.d;
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < a.dp; i += step) {       // (a thread reads back what it wrote)
    float u[8];
    load8(u_row + i, u);
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (i + j < a.d) ss = fmaf(u[j] - mean, u[j] - mean, ss);
  }
  const float rstd = 1.f / sqrtf(block_sum(ss, buf[3]) / (float)a.d + a.eps);
  const bool single = a.shift && r >= a.n_pre;
  T *hr = h + (size_t)blockIdx.x * a.dp, *st = nullptr;
  bool fresh = true;
  if (single) {
    st = static_cast<T*>(a.state) + (size_t)a.slot[a.row_seq[r]] * a.dp;
    fresh = a.pos[r] == 0;
  } else if (a.shift) {
    hr = static_cast<T*>(a.before) + (size_t)r * a.dp;
  }
  for (int i = threadIdx.x * 8; i < a.dp; i += step) {
    float u[8], w[8], b[8];
    load8(u_row + i, u);
    load8(a.w + i, w);
    load8(a.b + i, b);
#pragma unroll
    for (int j = 0; j < 8; ++j) u[j] = fmaf((u[j] - mean) * rstd, w[j], b[j]);
    if (single) {
      float p[8] = {}, f[8];
      if (!fresh) load8(st + i, p);
      store8(st + i, u);
      load8(a.shift + i, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float v = round_as(u[j], hr);
        u[j] = fmaf(p[j] - v, f[j], v);
      }
    }
    store8(hr + i, u);
  }
}

template <typename T>
__global__ void __launch_bounds__(ST_THREADS)
hy_shift_kernel(const T* __restrict__ in, T* __restrict__ out, const float* __restrict__ shift, T* __restrict__ state,
                const int* __restrict__ row_seq, const int* __restrict__ seq_row0, const int* __restrict__ seq_pos0,
                const int* __restrict__ seq_slot, int dp) {
  const int r = blockIdx.x, seq = row_seq[r];
  const bool first = r == seq_row0[seq], fresh = first && seq_pos0[seq] == 0;
  T* st = state + (size_t)seq_slot[seq] * dp;
  const T *cur = in + (size_t)r * dp, *last = in + (size_t)(seq_row0[seq + 1] - 1) * dp, *before = first ? st : cur - dp;
  for (int i = threadIdx.x * 8; i < dp; i += blockDim.x * 8) {
    float f[8], p[8] = {}, s[8];
    load8(cur + i, f);
    if (!fresh) load8(before + i, p);
    load8(shift + i, s);
#pragma unroll
    for (int j = 0; j < 8; ++j) s[j] = fmaf(p[j] - f[j], s[j], f[j]);
    store8(out + (size_t)r * dp + i, s);
    if (first) {
      load8(last + i, f);
      store8(st + i, f);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(ST_THREADS)
hy_gelu_kernel(const T* __restrict__ in, int ldi, T* __restrict__ out, int ldo, int n) {
  const int i = (blockIdx.y * ST_THREADS + threadIdx.x) * 8;
  if (i >= n) return;
  float f[8];
  load8(in + (size_t)blockIdx.x * ldi + i, f);
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = gelu_as<T>(f[j]);
  store8(out + (size_t)blockIdx.x * ldo + i, f);
}

__global__ void __launch_bounds__(ST_THREADS) hy_cap_kernel(float* __restrict__ x, long n, float cap) {
  const long i = ((long)blockIdx.x * ST_THREADS + threadIdx.x) * 4;
  if (i >= n) return;
  float4 v = *reinterpret_cast<float4*>(x + i);
  v.x = cap * tanhf(v.x / cap);
  v.y = cap * tanhf(v.y / cap);
  v.z = cap * tanhf(v.z / cap);
  v.w = cap * tanhf(v.w / cap);
  *reinterpret_cast<float4*>(x + i) = v;
}

static int row_threads(int dp) {
  const int t = (dp / 8 + 31) & ~31;
  return t > ST_THREADS ? ST_THREADS : t;
}

template <typename T, int S>
static int launch_streams_s(const StreamArgs& a, void* h, int n, cudaStream_t s) {
  static PerDeviceOnce once;
  const size_t smem = (size_t)a.dp * 4;
  if (smem > 200 * 1024) return BB_ESIZE;
  if (smem > 40 * 1024) {
    const cudaError_t e = ensure_dyn_smem(once, hy_streams_kernel<T, S>, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
  }
  hy_streams_kernel<T, S><<<n, row_threads(a.dp), smem, s>>>(a, static_cast<T*>(h));
  return (int)cudaGetLastError();
}
template <typename T>
static int launch_streams(const StreamArgs& a, void* h, int n, cudaStream_t s) {
  if (a.s <= 1) return launch_streams_s<T, 1>(a, h, n, s);
  if (a.s <= 2) return launch_streams_s<T, 2>(a, h, n, s);
  if (a.s <= 4) return launch_streams_s<T, 4>(a, h, n, s);
  if (a.s <= 8) return launch_streams_s<T, 8>(a, h, n, s);
  return a.s <= 16 ? launch_streams_s<T, 16>(a, h, n, s) : BB_ESIZE;
}

}  // namespace bb

using namespace bb;

// Start of a sublayer.  `before`: the layer whose sublayer fq (0 mixer, 1 feed-forward) has just run (null: the
// embedding); `next`: the layer whose sublayer tq starts (null: the rows whose logits are asked for -> hn, or with `all`
// every row's sum of streams -> trace).
BB_API int bb_hy_streams(const BbHyCfg* c, const BbHyLayer* before, int fq, const BbHyLayer* next, int tq, const BbHyWork* w,
                         const BbHyBatch* b, int all, float* trace, void* stream) {
  StreamArgs a{};
  const int n = next || all ? b->n : b->n_want;
  if (n <= 0) return BB_OK;
  a.x = w->x;
  a.rows = next || all ? nullptr : b->want;
  a.tok = b->tok;
  a.emb = before ? nullptr : c->embed;
  a.emb_scale = c->embed_scale;
  a.vocab = c->vocab;
  if (before) {
    a.from = before->hc[fq];
    if (fq == 1 && before->n_experts > 0) {
      a.ex_out = w->ex_out;
      a.pair_row = w->pair_row;
      a.pair_w = before->weigh_input ? nullptr : w->pair_w;
      a.top = before->top;
    } else {
      a.y32 = hy_sums_y(*c, b->n);
      a.ya = a.y32 ? w->ya32 : w->ya;
      if (fq == 0 && before->beside) {
        a.yb = a.y32 ? w->yb32 : w->yb;
        a.gain_a = before->out_gain;
        a.gain_b = before->beside->out_gain;
      }
    }
  }
  if (next && hy_sums_y(*c, b->n) && (tq == 0 || next->n_experts == 0)) {
    a.zero_a = w->ya32;
    a.zero_b = tq == 0 && next->beside ? w->yb32 : nullptr;
  }
  a.to = next ? next->hc[tq] : nullptr;
  a.w = next ? (tq ? next->norm2 : next->norm) : c->final_norm;
  a.b = next ? (tq ? next->norm2_b : next->norm_b) : c->final_norm_b;
  a.s = c->streams;
  a.write = next != nullptr;
  a.d = c->width;
  a.dp = c->dp;
  a.eps = c->eps;
  a.counts = w->ex_count;
  a.n_counts = next && tq == 1 ? next->n_experts : 0;
  a.trace = trace;
  if (next && tq == 0 && next->shift) {
    a.shift = next->shift;
    a.state = next->shift_state;
    a.before = w->h2;
    a.row_seq = b->row_seq;
    a.slot = b->seq_slot;
    a.pos = b->pos;
    a.n_pre = b->n_pre;
  }
  void* h = next ? w->h : w->hn;
  if (all && !next) h = w->h;
  return c->dtype ? launch_streams<float>(a, h, n, (cudaStream_t)stream) : launch_streams<__nv_bfloat16>(a, h, n, (cudaStream_t)stream);
}

// Shifted inputs of the prompt portions' rows.
BB_API int bb_hy_shift(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  if (b->n_pre <= 0 || !L->shift) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
#define BB_SHIFT(T)                                                                                                      \
  hy_shift_kernel<T><<<b->n_pre, row_threads(c->dp), 0, s>>>(static_cast<const T*>(w->h2), static_cast<T*>(w->h), L->shift, \
                                                             static_cast<T*>(L->shift_state), b->row_seq, b->seq_row0,   \
                                                             b->seq_pos0, b->seq_slot, c->dp)
  if (c->dtype) BB_SHIFT(float);
  else BB_SHIFT(__nv_bfloat16);
#undef BB_SHIFT
  return (int)cudaGetLastError();
}

// gelu of the layer's up projection (in the first columns of w->proj) -> the first columns of w->cat; the bf16 step has it in
// the projection's epilogue.
BB_API int bb_hy_gelu(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, int n, void* stream) {
  if (n <= 0) return BB_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const dim3 grid(n, (L->up.n / 8 + ST_THREADS - 1) / ST_THREADS);
  if (!c->dtype) return BB_EARG;
  hy_gelu_kernel<float><<<grid, ST_THREADS, 0, s>>>(static_cast<const float*>(w->proj), w->ld_proj, static_cast<float*>(w->cat),
                                                    w->ld_cat, L->up.n);
  return (int)cudaGetLastError();
}

BB_API int bb_hy_cap(const BbHyCfg* c, const BbHyWork* w, int n, void* stream) {
  if (n <= 0 || c->logit_cap <= 0.f) return BB_OK;
  const long total = (long)n * c->vocabp;
  hy_cap_kernel<<<(int)((total / 4 + ST_THREADS - 1) / ST_THREADS), ST_THREADS, 0, (cudaStream_t)stream>>>(w->logits, total, c->logit_cap);
  return (int)cudaGetLastError();
}

// Gated linear recurrence per channel (fp32 state; bf16 or fp32 projections, convolution and gates' maps):
//   r = sigmoid(gate + bias), i = sigmoid(gate + bias), log a = -lam r,
//   S <- a S + sqrt(1 - a^2) i u,   output S gelu(y + bias).
// a is carried as e = a - 1: where a is close to one its rounding to 32 bits would change the rate of a slow
// decay by 2^-25 / (1 - a), which long sequences show.  1 - a^2 = -e (2 + e).
//   hy_rglru_scan    prompt portions: a block owns 64 channels of a sequence and takes 128 tokens at a time,
//                    eight to a warp; the warps' (product of a, local S) pairs are chained through shared memory
//   hy_rglru_step    one token per sequence, one thread per two channels
// Both write the sequence's last taps - 1 raw convolution inputs into its slot (the convolution ran before).
// State: [slot][channel] fp32; a sequence at position 0 starts from zeros whatever its slot holds.
#include "../common/host.hpp"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

// Two channels as they are stored.
template <typename T>
struct alignas(sizeof(T) * 2) Pair {
  T v[2];
  __device__ __forceinline__ float2 f() const { return make_float2(to_f(v[0]), to_f(v[1])); }
};
template <typename T>
__device__ __forceinline__ Pair<T> raw_pair(const T* p) {
  return *reinterpret_cast<const Pair<T>*>(p);
}
template <typename T>
__device__ __forceinline__ float2 load_pair(const T* p) {
  return raw_pair(p).f();
}
template <typename T>
__device__ __forceinline__ void store_pair(T* p, float a, float b) {
  Pair<T> q;
  q.v[0] = from_f<T>(a);
  q.v[1] = from_f<T>(b);
  *reinterpret_cast<Pair<T>*>(p) = q;
}

// Everything below is 32-bit; with bf16 storage exponentials and divisions are the hardware's (2^-22).
// e^-x - 1 for x >= 0
template <typename T>
__device__ __forceinline__ float decay_m1(float x) {
  if constexpr (sizeof(T) == 2) {
    // the series where the difference would cancel
    return x < 0.05f ? -x * fmaf(x, fmaf(x, fmaf(x, -1.f / 24.f, 1.f / 6.f), -0.5f), 1.f) : exp_hw(-x) - 1.f;
  } else {
    return expm1f(-x);
  }
}
template <typename T>
__device__ __forceinline__ float root_of(float x) {
  if constexpr (sizeof(T) == 2) return x * rsqrt_hw(fmaxf(x, 1e-37f));
  else return sqrtf(x);
}
// S after a token of (e, in); product of two decays
__device__ __forceinline__ float2 lru_apply(float2 e, float2 s, float2 in) {
  return make_float2(s.x + fmaf(e.x, s.x, in.x), s.y + fmaf(e.y, s.y, in.y));
}
__device__ __forceinline__ float2 lru_product(float2 p, float2 e) {
  return make_float2(p.x + fmaf(e.x, p.x, e.x), p.y + fmaf(e.y, p.y, e.y));
}

struct LruChannels {
  float2 yb, rb, ib, lam;
};
__device__ __forceinline__ LruChannels lru_channels(const BbHyLayer& L, int c) {
  auto two = [&](const float* p) { return *reinterpret_cast<const float2*>(p + c); };
  return {two(L.y_b), two(L.r_b), two(L.i_b), two(L.lam)};
}
// Raw values of a token and two channels -> decay (less one) and input of the recurrence.
template <typename T>
__device__ __forceinline__ void lru_token(const LruChannels& p, float2 r, float2 i, float2 u, float2& e, float2& in) {
  e = make_float2(decay_m1<T>(p.lam.x * sigmoid_as<T>(r.x + p.rb.x)), decay_m1<T>(p.lam.y * sigmoid_as<T>(r.y + p.rb.y)));
  in = make_float2(root_of<T>(-e.x * (2.f + e.x)) * sigmoid_as<T>(i.x + p.ib.x) * u.x,
                   root_of<T>(-e.y * (2.f + e.y)) * sigmoid_as<T>(i.y + p.ib.y) * u.y);
}

template <typename T>
__device__ __forceinline__ void keep_input(const BbHyLayer& L, const T* row, int c, int pos, int ctx, int slot) {
  const int keep = L.taps - 1;
  if (keep <= 0 || pos < ctx - keep) return;
  T* ring = static_cast<T*>(L.conv_state) + ((size_t)slot * keep + pos % keep) * L.chp + c;
  const float2 x = load_pair(row + L.off_xbc + c);
  store_pair(ring, x.x, x.y);
}

constexpr int LRU_WARPS = 16, LRU_T = 8;

template <typename T>
__global__ void __launch_bounds__(LRU_WARPS * 32)
hy_rglru_scan_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ u, int ldu,
                     const T* __restrict__ gates, int ldg, T* __restrict__ cat, int ldc, const __grid_constant__ BbHyBatch b) {
  __shared__ float2 chain[2][LRU_WARPS][2][32];      // [buffer][warp][product of a | local S][lane]
  const int seq = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 64 + lane * 2;
  const bool live = c < L.chp;
  const int cc = live ? c : 0;
  const int r0 = b.seq_row0[seq], n = b.seq_row0[seq + 1] - r0, slot = b.seq_slot[seq], pos0 = b.seq_pos0[seq];
  const int ctx = pos0 + n;
  const int g0 = (cc / L.bwp) * 2 * L.bwp + cc % L.bwp;
  const LruChannels ch = lru_channels(L, cc);
  float* state = L.ssm_state + (size_t)slot * L.chp + cc;
  float2 carry = pos0 == 0 ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(state);
  // a warp's tokens of the next step are on their way while it works on this one's
  Pair<T> rr[LRU_T], ii[LRU_T], uu[LRU_T], yy[LRU_T];
  auto fetch = [&](int tw) {
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) {
      const size_t row = r0 + min(tw + k, n - 1);
      rr[k] = raw_pair(gates + row * ldg + g0);
      ii[k] = raw_pair(gates + row * ldg + g0 + L.bwp);
      uu[k] = raw_pair(u + row * ldu + cc);
    }
  };
  fetch(warp * LRU_T);
  for (int t0 = 0, it = 0; t0 < n; t0 += LRU_WARPS * LRU_T, ++it) {
    const int tw = t0 + warp * LRU_T;
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) yy[k] = raw_pair(proj + (size_t)(r0 + min(tw + k, n - 1)) * ld + L.off_y + cc);
    float2 p[LRU_T], s[LRU_T];
    {
      float2 pa = make_float2(0.f, 0.f), sa = make_float2(0.f, 0.f);
#pragma unroll
      for (int k = 0; k < LRU_T; ++k) {
        float2 e, in;
        lru_token<T>(ch, rr[k].f(), ii[k].f(), uu[k].f(), e, in);
        if (tw + k >= n) e = in = make_float2(0.f, 0.f);      // past the end: nothing changes
        sa = lru_apply(e, sa, in);
        pa = lru_product(pa, e);
        p[k] = pa;
        s[k] = sa;
      }
    }
    fetch(tw + LRU_WARPS * LRU_T);
    chain[it & 1][warp][0][lane] = p[LRU_T - 1];
    chain[it & 1][warp][1][lane] = s[LRU_T - 1];
    __syncthreads();
    float2 mine = carry;
#pragma unroll
    for (int w = 0; w < LRU_WARPS; ++w) {
      if (w == warp) mine = carry;
      carry = lru_apply(chain[it & 1][w][0][lane], carry, chain[it & 1][w][1][lane]);
    }
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) {
      if (tw + k < n && live) {
        const size_t row = r0 + tw + k;
        const float2 yv = yy[k].f();
        const float2 st = lru_apply(p[k], mine, s[k]);
        store_pair(cat + row * ldc + cc, st.x * gelu_as<T>(yv.x + ch.yb.x), st.y * gelu_as<T>(yv.y + ch.yb.y));
        keep_input<T>(L, proj + row * ld, cc, pos0 + tw + k, ctx, slot);
      }
    }
  }
  if (warp == 0 && live) *reinterpret_cast<float2*>(state) = carry;
}

template <typename T>
__global__ void __launch_bounds__(128)
hy_rglru_step_kernel(const __grid_constant__ BbHyLayer L, const T* __restrict__ proj, int ld, const T* __restrict__ u, int ldu,
                     const T* __restrict__ gates, int ldg, T* __restrict__ cat, int ldc, const __grid_constant__ BbHyBatch b) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 2;
  if (c >= L.chp) return;
  const int seq = b.ns_pre + blockIdx.y;
  const size_t row = b.n_pre + blockIdx.y;
  const int pos = b.pos[row], slot = b.seq_slot[seq];
  const int g0 = (c / L.bwp) * 2 * L.bwp + c % L.bwp;
  float* state = L.ssm_state + (size_t)slot * L.chp + c;
  const float2 old = *reinterpret_cast<const float2*>(state);
  const float2 yv = load_pair(proj + row * ld + L.off_y + c);
  const LruChannels ch = lru_channels(L, c);
  float2 e, in;
  lru_token<T>(ch, load_pair(gates + row * ldg + g0), load_pair(gates + row * ldg + g0 + L.bwp), load_pair(u + row * ldu + c), e, in);
  const bool fresh = pos == 0;
  const float2 s = fresh ? in : lru_apply(e, old, in);
  *reinterpret_cast<float2*>(state) = s;
  store_pair(cat + row * ldc + c, s.x * gelu_as<T>(yv.x + ch.yb.x), s.y * gelu_as<T>(yv.y + ch.yb.y));
  keep_input<T>(L, proj + row * ld, c, pos, pos + 1, slot);
}

template <typename T>
static int launch_rglru(const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  const T *proj = static_cast<const T*>(w.proj), *u = static_cast<const T*>(w.xbc), *g = static_cast<const T*>(w.aux);
  T* cat = static_cast<T*>(w.cat);
  if (b.ns_pre > 0)
    hy_rglru_scan_kernel<T><<<dim3((L.chp + 63) / 64, b.ns_pre), LRU_WARPS * 32, 0, s>>>(L, proj, w.ld_proj, u, w.ld_xbc, g,
                                                                                         w.ld_aux, cat, w.ld_cat, b);
  if (b.ns > b.ns_pre)
    hy_rglru_step_kernel<T><<<dim3((L.chp + 255) / 256, b.ns - b.ns_pre), 128, 0, s>>>(L, proj, w.ld_proj, u, w.ld_xbc, g,
                                                                                       w.ld_aux, cat, w.ld_cat, b);
  return (int)cudaGetLastError();
}

}  // namespace bb

using namespace bb;

// Recurrence of every row of the step (w->xbc: convolution outputs, w->aux: gate maps) -> w->cat.
BB_API int bb_hy_rglru(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  return c->dtype ? launch_rglru<float>(*L, *w, *b, (cudaStream_t)stream)
                  : launch_rglru<__nv_bfloat16>(*L, *w, *b, (cudaStream_t)stream);
}

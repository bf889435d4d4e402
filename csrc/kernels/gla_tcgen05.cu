// Gated linear attention of prompt portions in chunks of 128 tokens on the tensor cores (bf16 projections, fp32 state), a
// decay for every token and key channel.  With L the running sum of the decays' logarithms inside a chunk, L_C its last
// value and S the state before the chunk, channel by channel:
//   S' = e^L_C S + (k e^(L_C - L))^T v
//   o  = (q e^(L - m)) (e^m S)  +  mask((q e^(L - m)) (k e^(m - L))^T) v,     m = L_C / 2
// so the decays go into the operands and the products are plain ones; what is not masked has L_i - L_j <= 0.
//   gla_parts     per chunk: L (kept for the outputs) and what the chunk adds to the state
//   gla_carry     per state element: the state before every chunk, in the parts' place, and the state behind the last
//   gla_outputs   per chunk: outputs, head norm, gain and gate
// Chunks of one sequence do not wait for one another but in gla_carry.  Operands that are not bf16 by nature (scaled
// queries and keys, the state, the masked scores) are two bf16 terms each.  A chunk in which some channel decays by more
// than e^-120 marks its (sequence, head): that is left to the scan (hy_linear_scan), whatever the other chunks hold.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../common/split.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int GL_THREADS = 256, GL_SUB = 128 * 128, GL_N = 64;   // a sub-tile: 128 rows of 64 bf16; key channels at most
constexpr float GL_LIMIT = 120.f;

// Where the chunks of a sequence start among all: no two sequences overlap, as ceil(len / 128) <= len / 128 + 1.
__device__ __forceinline__ int chunk_slot0(const BbHyBatch& b, int seq) { return b.seq_row0[seq] / 128 + seq; }

__device__ __forceinline__ bool left_to_scan(const int* flags, const BbHyBatch& b, int seq, int heads, int h) {
  const int n = (b.seq_row0[seq + 1] - b.seq_row0[seq] + 127) / 128, s0 = chunk_slot0(b, seq);
  bool any = false;
  for (int c = 0; c < n; ++c) any |= flags[(s0 + c) * heads + h] != 0;
  return any;
}

// Two terms of two values into columns c, c + 1 (c even) of a row of two swizzled tiles.
__device__ __forceinline__ void put_split(uint8_t* hi, uint8_t* lo, int row, int c, float a, float b) {
  const float2 t = split_pair(a, b);
  const int o = swizzled(row, c & ~7, GL_SUB) + (c & 7) * 2;
  *reinterpret_cast<float*>(hi + o) = t.x;
  *reinterpret_cast<float*>(lo + o) = t.y;
}
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

template <int PP>
struct GlaParts {
  static constexpr int PSUB = PP / 64;
  static constexpr int OFF_K = 0, OFF_V = 2 * GL_SUB, OFF_E = OFF_V + PSUB * GL_SUB;   // keys, two terms; values; sums, barriers
  static constexpr int SMEM = OFF_E + 8 * 64 * 4 + 64;
};

template <int PP>
__global__ void __launch_bounds__(GL_THREADS, 2)
gla_parts_kernel(const __grid_constant__ CUtensorMap tmV, const __grid_constant__ BbHyLayer L,
                 const __nv_bfloat16* __restrict__ proj, int ld, const float* __restrict__ z, float* __restrict__ logs, int ldz,
                 float* __restrict__ parts, int* __restrict__ flags, const __grid_constant__ BbHyBatch b, int* err) {
  using Cfg = GlaParts<PP>;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t *sK = smem + Cfg::OFF_K, *sV = smem + Cfg::OFF_V;
  float2* s_sum = reinterpret_cast<float2*>(smem + Cfg::OFF_E);    // [8][32]
  uint64_t *b_v = reinterpret_cast<uint64_t*>(s_sum + 256), *b_s = b_v + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(b_v + 2);
  const int seq = b.tile_seq[blockIdx.x], c = b.tile_qt[blockIdx.x], h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r0 = b.seq_row0[seq] + c * 128, valid = min(128, b.seq_row0[seq + 1] - r0);
  const int slot = (chunk_slot0(b, seq) + c) * L.heads + h;
  if (threadIdx.x == 0) {
    mbar_init(b_v, 1);
    mbar_init(b_s, 1);
    mbar_fence_init();
    mbar_expect_tx(b_v, Cfg::PSUB * GL_SUB);
    for (int s = 0; s < Cfg::PSUB; ++s) tma_load_3d(sV + s * GL_SUB, &tmV, b_v, s * 64, r0, h);
  }
  __syncwarp();
  if (warp == 0) {
    tmem_alloc(tmem_slot, PP);
    tmem_relinquish();
  }
  // two channels of 16 tokens to a thread: logarithms of the decays and their running sum
  constexpr int TOK = 128 / (GL_THREADS / 32);
  const int ch = lane * 2, t0 = warp * TOK;
  const bool in = ch < L.np;                         // (channels past the true number have no keys and decay by nothing)
  float2 lg[TOK], sum = make_float2(0.f, 0.f);
  {
    const float* zr = z + (size_t)(r0 + t0) * ldz + h * L.np + ch;
#pragma unroll
    for (int t = 0; t < TOK; ++t)
      lg[t] = in && t0 + t < valid ? *reinterpret_cast<const float2*>(zr + (size_t)t * ldz) : make_float2(0.f, 0.f);
    const float2 bias = in ? *reinterpret_cast<const float2*>(L.w0 + h * L.np + ch) : make_float2(0.f, 0.f);
    auto log_decay = [&](float x) { return -L.decay_root * (fmaxf(-x, 0.f) + log1pf(expf(-fabsf(x)))); };
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
      if (t0 + t < valid) {
        if (ch < L.n) sum.x += log_decay(lg[t].x + bias.x);
        if (ch + 1 < L.n) sum.y += log_decay(lg[t].y + bias.y);
      }
      lg[t] = sum;
    }
  }
  s_sum[warp * 32 + lane] = sum;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  float2 base = make_float2(0.f, 0.f), all = base;
#pragma unroll
  for (int s = 0; s < GL_THREADS / 32; ++s) {
    if (s == warp) base = all;
    all.x += s_sum[s * 32 + lane].x;
    all.y += s_sum[s * 32 + lane].y;
  }
  {
    const __nv_bfloat16* kr = proj + (size_t)(r0 + t0) * ld + L.off_kk + h * L.np + ch;
    float* lr = logs + (size_t)(r0 + t0) * ldz + h * L.np + ch;
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
      float2 k = make_float2(0.f, 0.f);
      if (in && t0 + t < valid) {
        const float2 l = make_float2(base.x + lg[t].x, base.y + lg[t].y);
        *reinterpret_cast<float2*>(lr + (size_t)t * ldz) = l;
        k = load_pair(kr + (size_t)t * ld);
        k.x *= expf(all.x - l.x);
        k.y *= expf(all.y - l.y);
      }
      put_split(sK, sK + GL_SUB, t0 + t, ch, k.x, k.y);
    }
  }
  fence_proxy_async_smem();
  bool ok = (smem_u32(smem) & 1023u) == 0 && mbar_wait(b_v, 0);
  const int strong = __syncthreads_or(fminf(all.x, all.y) < -GL_LIMIT);
  ok = __syncthreads_and(ok);
  if (threadIdx.x == 0) flags[slot] = strong;
  const uint32_t tm = *tmem_slot;
  if (ok && !strong) {
    if (threadIdx.x == 0) {
      constexpr uint32_t id = umma_idesc(1, 1, 1, 1, 1, 128, PP);
      const uint32_t aK = smem_u32(sK), aV = smem_u32(sV);
      tc_fence_after();
#pragma unroll
      for (int t = 0; t < 8; ++t)     // rows of the product: channels by their value, then by their remainder
        umma_f16_ss(tm, umma_smem_desc(aK + t * 2048, GL_SUB, 1024), umma_smem_desc(aV + t * 2048, GL_SUB, 1024), id, t != 0);
      umma_commit(b_s);
    }
    __syncwarp();
    ok = mbar_wait(b_s, 0);
    tc_fence_after();
    // the two halves of the rows are added up through shared memory (the keys are behind their products)
    constexpr int HC = PP / 2;
    const int row = (warp & 3) * 32 + lane, col0 = (warp >> 2) * HC;
    float* s_st = reinterpret_cast<float*>(sK);      // [64][PP], columns exclusive-or'ed with the row
    const uint32_t tS = tm + ((uint32_t)((warp & 3) * 32) << 16) + col0;
    ok = __syncthreads_and(ok);
    for (int part = 1; part >= 0; --part) {
      if (row / 64 == part) {
        const int n = row & 63;
#pragma unroll
        for (int c0 = 0; c0 < HC; c0 += 32) {
          uint32_t r[32];
          tmem_ld32(tS + c0, r);
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            float& s = s_st[n * PP + ((col0 + c0 + j) ^ (n & 31))];
            s = part ? __uint_as_float(r[j]) : s + __uint_as_float(r[j]);
          }
        }
      }
      __syncthreads();
    }
    float* dst = parts + (size_t)slot * L.n * L.p;
    for (int n = warp; ok && n < L.n; n += GL_THREADS / 32)
      for (int p = lane; p < L.p; p += 32) dst[(size_t)n * L.p + p] = s_st[n * PP + (p ^ (n & 31))];
  }
  if (!ok && threadIdx.x == 0) set_error(err, ERR_WAIT_EPILOGUE);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tm, PP);
  }
}

constexpr int GC_AHEAD = 8;      // chunks asked for ahead of their use

__global__ void __launch_bounds__(256)
gla_carry_kernel(const __grid_constant__ BbHyLayer L, const float* __restrict__ logs, int ldz, float* __restrict__ parts,
                 const int* __restrict__ flags, const __grid_constant__ BbHyBatch b) {
  const int seq = blockIdx.x, h = blockIdx.y, np = L.n * L.p, i = blockIdx.z * 256 + threadIdx.x;
  if (left_to_scan(flags, b, seq, L.heads, h) || i >= np) return;
  const int r0 = b.seq_row0[seq], r1 = b.seq_row0[seq + 1], n_chunks = (r1 - r0 + 127) / 128, n = i / L.p;
  float* state = L.ssm_state + ((size_t)b.seq_slot[seq] * L.heads + h) * np + i;
  float* part = parts + ((size_t)chunk_slot0(b, seq) * L.heads + h) * np + i;
  const size_t step = (size_t)L.heads * np;
  float s = b.seq_pos0[seq] == 0 ? 0.f : *state;
  for (int c0 = 0; c0 < n_chunks; c0 += GC_AHEAD) {
    float u[GC_AHEAD], l[GC_AHEAD];
#pragma unroll
    for (int a = 0; a < GC_AHEAD; ++a)
      if (c0 + a < n_chunks) {
        u[a] = part[(c0 + a) * step];
        l[a] = logs[(size_t)(min(r0 + (c0 + a + 1) * 128, r1) - 1) * ldz + h * L.np + n];
      }
#pragma unroll
    for (int a = 0; a < GC_AHEAD; ++a)
      if (c0 + a < n_chunks) {
        part[(c0 + a) * step] = s;
        s = fmaf(s, expm1f(l[a]), s) + u[a];
      }
  }
  *state = s;
}

template <int PP>
struct GlaOut {
  static constexpr int PSUB = PP / 64;
  static constexpr int OFF_Q = 0;                                  // queries, two terms; then the rows on their way out
  static constexpr int OFF_K = OFF_Q + 2 * GL_SUB;                 // keys, two terms; then values
  static constexpr int S_SUB = GL_SUB / 2;                         // 64 rows
  static constexpr int OFF_S = OFF_K + 2 * GL_SUB;                 // the state, two terms
  static constexpr int OFF_E = OFF_S + 2 * PSUB * S_SUB;           // [2][128] sums, barriers
  static constexpr int SMEM = OFF_E + 1024 + 64;
  static constexpr int COL_Y = 128, TMEM_COLS = 256;
};

template <int PP>
__global__ void __launch_bounds__(GL_THREADS, 2)
gla_outputs_kernel(const __grid_constant__ CUtensorMap tmV, const __grid_constant__ BbHyLayer L,
                   const __nv_bfloat16* __restrict__ proj, int ld, const float* __restrict__ logs, int ldz,
                   const float* __restrict__ parts, const int* __restrict__ flags, __nv_bfloat16* __restrict__ out, int ldo,
                   const __grid_constant__ BbHyBatch b, float eps, int* err) {
  using Cfg = GlaOut<PP>;
  constexpr int HC = PP / 2;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t *sQ = smem + Cfg::OFF_Q, *sK = smem + Cfg::OFF_K, *sS = smem + Cfg::OFF_S, *sSl = sS + Cfg::PSUB * Cfg::S_SUB;
  float* s_sum = reinterpret_cast<float*>(smem + Cfg::OFF_E);
  uint64_t *b_g = reinterpret_cast<uint64_t*>(s_sum + 256), *b_v = b_g + 1, *b_y = b_g + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(b_g + 3);
  const int seq = b.tile_seq[blockIdx.x], c = b.tile_qt[blockIdx.x], h = blockIdx.y;
  if (left_to_scan(flags, b, seq, L.heads, h)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = (warp & 3) * 32 + lane, half = warp >> 2;
  const int r0 = b.seq_row0[seq] + c * 128, valid = min(128, b.seq_row0[seq + 1] - r0);
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(b_g + i, 1);
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  const float* last = logs + (size_t)(r0 + valid - 1) * ldz + h * L.np;
  {
    constexpr int TOK = 128 / (GL_THREADS / 32);
    const int ch = lane * 2, t0 = warp * TOK;
    const bool in = ch < L.np;
    const float2 end = in ? *reinterpret_cast<const float2*>(last + ch) : make_float2(0.f, 0.f);
    const __nv_bfloat16* pr = proj + (size_t)(r0 + t0) * ld + h * L.np + ch;
    const float* lr = logs + (size_t)(r0 + t0) * ldz + h * L.np + ch;
#pragma unroll 8
    for (int t = 0; t < TOK; ++t) {
      float2 q = make_float2(0.f, 0.f), k = q;
      if (in && t0 + t < valid) {
        const float2 l = *reinterpret_cast<const float2*>(lr + (size_t)t * ldz);
        const float x = l.x - 0.5f * end.x, y = l.y - 0.5f * end.y;
        q = load_pair(pr + (size_t)t * ld + L.off_q);
        k = load_pair(pr + (size_t)t * ld + L.off_kk);
        q.x *= expf(x);
        q.y *= expf(y);
        k.x *= expf(-x);
        k.y *= expf(-y);
      }
      put_split(sQ, sQ + GL_SUB, t0 + t, ch, q.x, q.y);
      put_split(sK, sK + GL_SUB, t0 + t, ch, k.x, k.y);
    }
  }
  {
    const int n = threadIdx.x >> 2, col0 = (threadIdx.x & 3) * (PP / 4);
    const float* src = parts + ((size_t)(chunk_slot0(b, seq) + c) * L.heads + h) * L.n * L.p + (size_t)n * L.p;
    const float f = n < L.n ? expf(0.5f * last[n]) : 0.f;
    float v[PP / 4];
    if (n < L.n && (L.p & 3) == 0 && col0 + PP / 4 <= L.p) {
#pragma unroll
      for (int j = 0; j < PP / 4; j += 4) {
        const float4 x = *reinterpret_cast<const float4*>(src + col0 + j);
        v[j] = x.x * f; v[j + 1] = x.y * f; v[j + 2] = x.z * f; v[j + 3] = x.w * f;
      }
    } else {
#pragma unroll
      for (int j = 0; j < PP / 4; ++j) v[j] = n < L.n && col0 + j < L.p ? src[col0 + j] * f : 0.f;
    }
    store_split(sS, sSl, n, col0, v, Cfg::S_SUB);
  }
  fence_proxy_async_smem();
  tc_fence_before();
  bool ok = __syncthreads_and((smem_u32(smem) & 1023u) == 0);
  tc_fence_after();
  const uint32_t tm = *tmem_slot, tG = tm + ((uint32_t)((warp & 3) * 32) << 16), tY = tG + Cfg::COL_Y + half * HC;
  if (ok && threadIdx.x == 0) {
    constexpr uint32_t id_g = umma_idesc(1, 1, 1, 0, 0, 128, 128), id_y = umma_idesc(1, 1, 1, 0, 1, 128, PP);
    const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aS = smem_u32(sS), aSl = smem_u32(sSl);
    const int nk = (L.n + 15) / 16;
    // products of two terms each: value x value, remainder x value, value x remainder
    for (int t = 0; t < nk; ++t)
      for (int x = 0; x < 3; ++x)
        umma_f16_ss(tm, umma_smem_desc(aQ + (x == 1 ? GL_SUB : 0) + t * 32, 16, 1024),
                    umma_smem_desc(aK + (x == 2 ? GL_SUB : 0) + t * 32, 16, 1024), id_g, (t | x) != 0);
    for (int t = 0; t < nk; ++t)
      for (int x = 0; x < 3; ++x)
        umma_f16_ss(tm + Cfg::COL_Y, umma_smem_desc(aQ + (x == 1 ? GL_SUB : 0) + t * 32, 16, 1024),
                    umma_smem_desc((x == 2 ? aSl : aS) + t * 2048, Cfg::S_SUB, 1024), id_y, (t | x) != 0);
    umma_commit(b_g);
  }
  __syncwarp();
  ok = ok && mbar_wait(b_g, 0);
  tc_fence_after();
  // values into the keys' place; scores into registers before any thread writes over them
  ok = __syncthreads_and(ok);
  if (ok && threadIdx.x == 0) {
    mbar_expect_tx(b_v, Cfg::PSUB * GL_SUB);
    for (int s = 0; s < Cfg::PSUB; ++s) tma_load_3d(sK + s * GL_SUB, &tmV, b_v, s * 64, r0, h);
  }
  __syncwarp();
  if (ok) {
    uint32_t g0[32], g1[32];
    tmem_ld32(tG + half * 64, g0);
    tmem_ld32(tG + half * 64 + 32, g1);
    tmem_wait_ld();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const int lim = row - half * 64;       // columns j <= lim are in the past
    auto keep = [&](const uint32_t (&g)[32], int j0) {
      uint32_t hi[16], lo[16];
#pragma unroll
      for (int j = 0; j < 32; j += 2) {
        const float2 s = split_pair(j0 + j <= lim ? __uint_as_float(g[j]) : 0.f, j0 + j + 1 <= lim ? __uint_as_float(g[j + 1]) : 0.f);
        hi[j >> 1] = __float_as_uint(s.x);
        lo[j >> 1] = __float_as_uint(s.y);
      }
      tmem_st16(tG + half * 32 + (j0 >> 1), hi);
      tmem_st16(tG + 64 + half * 32 + (j0 >> 1), lo);
    };
    keep(g0, 0);
    keep(g1, 32);
    tmem_wait_st();
    tc_fence_before();
    ok = mbar_wait(b_v, 0);
    ok = __syncthreads_and(ok);
  }
  if (ok) {
    if (threadIdx.x == 0) {
      tc_fence_after();
      constexpr uint32_t id_y = umma_idesc(1, 1, 1, 0, 1, 128, PP);
      const uint32_t aV = smem_u32(sK);
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        const uint64_t dv = umma_smem_desc(aV + t * 2048, GL_SUB, 1024);
        umma_f16_ts(tm + Cfg::COL_Y, tm + t * 8, dv, id_y, 1);
        umma_f16_ts(tm + Cfg::COL_Y, tm + 64 + t * 8, dv, id_y, 1);
      }
      umma_commit(b_y);
    }
    __syncwarp();
    constexpr int VR = PP / 8, OUT_IT = 128 * VR / GL_THREADS;      // 16-byte pieces of a row; those of a thread
    bf16x8 gate[OUT_IT];
#pragma unroll
    for (int it = 0; it < OUT_IT; ++it) {
      const int i = threadIdx.x + it * GL_THREADS, rr = i / VR, q = i % VR;
      if (rr < valid && q * 8 < L.pp)
        gate[it] = *reinterpret_cast<const bf16x8*>(proj + (size_t)(r0 + rr) * ld + L.off_gg + h * L.pp + q * 8);
    }
    ok = mbar_wait(b_y, 0);
    tc_fence_after();
    __syncwarp();
    float o[HC], ss = 0.f;
#pragma unroll
    for (int j0 = 0; j0 < HC; j0 += 32) {
      uint32_t r[32];
      tmem_ld32(tY + j0, r);
      tmem_wait_ld();
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        o[j0 + j] = __uint_as_float(r[j]) * L.q_scale;
        ss = fmaf(o[j0 + j], o[j0 + j], ss);
      }
    }
    s_sum[half * 128 + row] = ss;
    ok = __syncthreads_and(ok);
    const float rstd = 1.f / sqrtf((s_sum[row] + s_sum[128 + row]) / (float)L.p + eps);
#pragma unroll
    for (int q = 0; q < HC / 8; ++q) {
      float x[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = o[q * 8 + j] * rstd;
      store8(reinterpret_cast<__nv_bfloat16*>(sQ + swizzled(row, half * HC + q * 8, GL_SUB)), x);
    }
    __syncthreads();
#pragma unroll
    for (int it = 0; it < OUT_IT; ++it) {
      const int i = threadIdx.x + it * GL_THREADS, rr = i / VR, q = i % VR, col = h * L.pp + q * 8;
      if (ok && rr < valid && q * 8 < L.pp) {
        float f[8], g[8], w[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sQ + swizzled(rr, q * 8, GL_SUB)), f);
        unpack8(gate[it], g);
        load8(L.gnorm + col, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= w[j] * silu_as<__nv_bfloat16>(g[j]);
        store8(out + (size_t)(r0 + rr) * ldo + col, f);
      }
    }
  }
  if (!ok && threadIdx.x == 0) set_error(err, ERR_WAIT_EPILOGUE);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tm, Cfg::TMEM_COLS);
  }
}

template <int PP>
static int launch_gla(const CUtensorMap& tmV, const BbHyCfg& c, const BbHyLayer& L, const BbHyWork& w, const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once_p, once_o;
  cudaError_t e = ensure_dyn_smem(once_p, gla_parts_kernel<PP>, GlaParts<PP>::SMEM);
  if (e != cudaSuccess) return (int)e;
  e = ensure_dyn_smem(once_o, gla_outputs_kernel<PP>, GlaOut<PP>::SMEM);
  if (e != cudaSuccess) return (int)e;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(w.proj);
  float* logs = w.f32 + L.heads * L.np;
  int* err = device_error_word();
  const dim3 grid(b.n_tiles, L.heads);
  gla_parts_kernel<PP><<<grid, GL_THREADS, GlaParts<PP>::SMEM, s>>>(tmV, L, proj, w.ld_proj, w.f32, logs, w.ld_f32, w.chunks,
                                                                    w.chunk_flags, b, err);
  gla_carry_kernel<<<dim3(b.ns_pre, L.heads, (L.n * L.p + 255) / 256), 256, 0, s>>>(L, logs, w.ld_f32, w.chunks, w.chunk_flags, b);
  gla_outputs_kernel<PP><<<grid, GL_THREADS, GlaOut<PP>::SMEM, s>>>(tmV, L, proj, w.ld_proj, logs, w.ld_f32, w.chunks, w.chunk_flags,
                                                                    static_cast<__nv_bfloat16*>(w.cat), w.ld_cat, b, c.eps, err);
  return (int)cudaGetLastError();
}

}  // namespace bb

// Prompt portions, bf16, from z in the first columns of w->f32 (the next ones get the logarithms' sums): recurrence, norm
// and gate -> w->cat, but for the (sequence, head) pairs marked in w->chunk_flags.  BB_ESIZE for heads above 64 key or 128
// value channels, constant decays, and more chunks than the scratch holds.
BB_API int bb_gla_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  using namespace bb;
  if (b->ns_pre <= 0) return BB_OK;
  const long slots = b->n_pre / 128 + b->ns_pre;
  if (c->dtype || !L->w2.w || !L->gnorm || L->np > GL_N || L->pp > 128 || w->ld_f32 < 2 * L->heads * L->np ||
      slots * L->heads * L->n * L->p > w->chunk_floats || slots * L->heads > w->chunk_marks)
    return BB_ESIZE;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(w->proj);
  CUtensorMap tmV;
  const int rc = make_tmap_3d(&tmV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, proj + L->off_vv, L->pp, b->n_pre, L->heads,
                              (uint64_t)w->ld_proj * 2, (uint64_t)L->pp * 2, 64, 128);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return L->p <= 64 ? launch_gla<64>(tmV, *c, *L, *w, *b, s) : launch_gla<128>(tmV, *c, *L, *w, *b, s);
}

// State-space recurrence of prompt portions in chunks of 128 tokens on the tensor cores (bf16 inputs,
// fp32 accumulation and state).  One CTA per (sequence, head) walks its portion chunk by chunk:
//
//   G = C B^T                                  128 x 128, K = state size
//   Y = exp(cum_i) (C S)  +  W X               W_ij = G_ij exp(cum_i - cum_j) dt_j for j <= i, else 0
//   S = exp(cum_last) S + B^T X'               X'_j = exp(cum_last - cum_j) dt_j x_j
//   y_i = Y_i + D x_i
//
// with cum the running sum of a dt inside the chunk.  The state S lives in TMEM as an fp32 accumulator
// from the first chunk to the last.  The operands that are not bf16 by nature - the weights W, the
// scaled inputs X' and the state S as an operand - go through the tensor core as two bf16 terms each
// (value and remainder, 16 bits of mantissa), so the recurrence keeps its 32-bit character.
//
// With few (sequence, head) pairs a portion is cut into segments of whole chunks that run side by side:
// a first launch (LOCAL) computes what each segment adds to the state on its own, and its decay; the
// segments of the main launch then start from the state carried in, decayed and summed over the segments
// before them.
//
// 256 threads: TMEM lane = token (or state row), two warpgroups share a row's columns.  Thread 0 issues
// TMA and MMA.  The phases of a chunk are separated by block barriers; with head sizes up to 64 two CTAs
// share an SM (113 KB of shared memory, 256 TMEM columns each) and fill each other's gaps.
// TMEM: G, then W as packed bf16 (value in its first 64 columns, remainder in the others); Y; S.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int SSD_THREADS = 256;
constexpr int SSD_SUB = 128 * 128;   // one swizzled sub-tile: 128 rows of 64 bf16

template <int PP>
struct SsdCfg {
  static constexpr int PSUB = PP / 64;
  static constexpr int OFF_C = 0;                               // 2 sub-tiles
  static constexpr int OFF_B = OFF_C + 2 * SSD_SUB;             // 2
  static constexpr int OFF_X = OFF_B + 2 * SSD_SUB;             // PSUB
  static constexpr int OFF_S = OFF_X + PSUB * SSD_SUB;          // 2 PSUB: S as two terms, then X' as two terms
  static constexpr int OFF_E = OFF_S + 2 * PSUB * SSD_SUB;      // 128 floats, 8 partial sums, barriers
  static constexpr int SMEM = OFF_E + 1024;
  // TMEM columns.  The state product of a chunk leaves its two terms side by side: the first added to S,
  // the second in T right behind it (one 2 PP wide MMA per step instead of two, which cost the same each).
  // With PP = 64 T lies over the first half of W, whose products are issued before.
  static constexpr int COL_G = PP == 64 ? 128 : 0, COL_Y = PP == 64 ? 0 : 128, COL_S = PP == 64 ? 64 : 256;
  static constexpr int COL_T = COL_S + PP;
  static constexpr int TMEM_COLS = PP == 64 ? 256 : 512;
};

__device__ __forceinline__ float2 split_pair(float a, float b) {
  // packed bf16 pair of the values, packed pair of what rounding left over
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  return make_float2(__uint_as_float(*reinterpret_cast<const uint32_t*>(&h)),
                     __uint_as_float(*reinterpret_cast<const uint32_t*>(&l)));
}

// 32 fp32 values of row `row`, columns col0.. (a multiple of 8), as two bf16 terms into two swizzled tiles.
__device__ __forceinline__ void store_split(uint8_t* hi, uint8_t* lo, int row, int col0, const float (&v)[32]) {
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 t = split_pair(v[q * 8 + 2 * k], v[q * 8 + 2 * k + 1]);
      h[k] = __float_as_uint(t.x);
      l[k] = __float_as_uint(t.y);
    }
    const int col = col0 + q * 8;
    const int o = (col >> 6) * SSD_SUB + row * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4);
    *reinterpret_cast<uint4*>(hi + o) = make_uint4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<uint4*>(lo + o) = make_uint4(l[0], l[1], l[2], l[3]);
  }
}

template <int PP, bool LOCAL>
__global__ void __launch_bounds__(SSD_THREADS, PP == 64 ? 2 : 1)
ssd_chunk_kernel(const __grid_constant__ CUtensorMap tmBC, const __grid_constant__ CUtensorMap tmX,
                 const __grid_constant__ BbHyLayer L, const float* __restrict__ dt, int lddt,
                 __nv_bfloat16* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b, int segs,
                 float* __restrict__ seg, int* err) {
  using Cfg = SsdCfg<PP>;
  constexpr int PSUB = Cfg::PSUB, HC = PP / 2;   // HC: Y / S / X columns of a thread
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sC = smem + Cfg::OFF_C;
  uint8_t* sB = smem + Cfg::OFF_B;
  uint8_t* sX = smem + Cfg::OFF_X;
  uint8_t* sS = smem + Cfg::OFF_S;
  uint8_t* sSl = sS + PSUB * SSD_SUB;
  float* s_e = reinterpret_cast<float*>(smem + Cfg::OFF_E);   // [128]
  float* s_part = s_e + 128;                                  // [8] warp sums of the coming chunk
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_part + 8);
  uint64_t *b_tma = bars, *b_gy = bars + 1, *b_y = bars + 2, *b_s = bars + 3;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 4);

  const int seq = blockIdx.x, h = blockIdx.y, grp = h / (L.heads / L.groups);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = (warp & 3) * 32 + lane, half = warp >> 2;
  const uint32_t lane_sel = (uint32_t)((warp & 3) * 32) << 16;
  const int r0 = b.seq_row0[seq], len = b.seq_row0[seq + 1] - r0, slot = b.seq_slot[seq];
  const int n_chunks = (len + 127) / 128;
  const int nsub = (L.n + 63) / 64, nk = (L.n + 15) / 16;
  const float a2 = L.a[h] * 1.4426950408889634f, D = L.d_skip[h];
  float* state = L.ssm_state + ((size_t)slot * L.heads + h) * L.n * L.p;

  // this CTA's chunks, and the scratch of its (sequence, head): segment states, the state carried in, decays
  const int z = blockIdx.z, per = (n_chunks + segs - 1) / segs, z_last = (n_chunks - 1) / per;
  if (z > z_last || (LOCAL && z > 0 && z == z_last)) return;
  const int ch0 = z * per, ch1 = LOCAL && z == z_last ? ch0 : min(n_chunks, ch0 + per);
  const size_t np = (size_t)L.n * L.p;
  float* sg = seg + ((size_t)seq * L.heads + h) * ((segs + 1) * np + segs);
  float* s_carry = sg + segs * np;
  float* s_dec = s_carry + np;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(bars + i, 1);
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  if (nsub == 1) {   // the state rows above 64 that the 128-row accumulator has anyway stay zero
    for (int i = threadIdx.x; i < SSD_SUB / 16; i += SSD_THREADS)
      reinterpret_cast<uint4*>(sB + SSD_SUB)[i] = make_uint4(0, 0, 0, 0);
    fence_proxy_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = *tmem_slot;
  const uint32_t tG = tm + Cfg::COL_G + lane_sel, tY = tm + Cfg::COL_Y + lane_sel + half * HC, tS = tm + Cfg::COL_S + lane_sel + half * HC,
                 tT = tm + Cfg::COL_T + lane_sel + half * HC;
  // The state between memory and TMEM goes through the operand tiles' place as fp32 [128][PP], columns
  // exclusive-or'ed with the row: a warp moves whole rows of memory, a thread reads or writes its own row.
  float* s_st = reinterpret_cast<float*>(sS);
  {
    const bool fresh = b.seq_pos0[seq] == 0;
#pragma unroll 4
    for (int n = warp; n < 128; n += SSD_THREADS / 32) {
#pragma unroll
      for (int p0 = 0; p0 < PP; p0 += 32) {
        const int p = p0 + lane;
        const size_t i = (size_t)n * L.p + p;
        float v = 0.f;
        if (n < L.n && p < L.p) {
          if (LOCAL) {
            if (z == 0) {
              v = fresh ? 0.f : state[i];
              s_carry[i] = v;      // the main launch may write the slot before its first segment reads it
            }
          } else if (segs == 1) {
            v = fresh ? 0.f : state[i];
          } else if (z == 0) {
            v = s_carry[i];
          } else {
            v = sg[i];             // (it includes the state carried in)
            for (int k = 1; k < z; ++k) v = fmaf(v, s_dec[k], sg[k * np + i]);
          }
        }
        s_st[n * PP + (p ^ (n & 31))] = v;
      }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < HC; c += 32) {
      uint32_t r[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(s_st[row * PP + ((half * HC + c + j) ^ (row & 31))]);
      tmem_st32(tS + c, r);
    }
    tmem_wait_st();
  }

  // step sizes of a chunk and their running sum inside a warp (log2 units), a chunk ahead of their use;
  // both warpgroups scan the same 128 tokens
  float d_next = 0.f, cum_next = 0.f;
  auto load_dt = [&](int ch) {
    const int i = ch * 128 + row;
    d_next = i < len ? dt[(size_t)(r0 + i) * lddt + h] : 0.f;
  };
  auto scan_dt = [&]() {
    cum_next = a2 * d_next;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, cum_next, o);
      if (lane >= o) cum_next += v;
    }
    if (lane == 31) s_part[warp] = cum_next;
  };
  load_dt(ch0);
  scan_dt();
  __syncthreads();

  bool ok = (smem_u32(smem) & 1023u) == 0;
  if (!ok && threadIdx.x == 0) set_error(err, ERR_BAD_ARG);
  float decay_log = 0.f;
  for (int ch = ch0; ch < ch1 && ok; ++ch) {
    const uint32_t ph = (ch - ch0) & 1;
    const int c0 = r0 + ch * 128, valid = min(128, len - ch * 128);
    if (threadIdx.x == 0) {
      mbar_expect_tx(b_tma, ((LOCAL ? 1 : 2) * nsub + PSUB) * SSD_SUB);
      for (int s = 0; s < nsub; ++s) {
        if (!LOCAL) tma_load_3d(sC + s * SSD_SUB, &tmBC, b_tma, s * 64, c0, L.groups + grp);
        tma_load_3d(sB + s * SSD_SUB, &tmBC, b_tma, s * 64, c0, grp);
      }
      for (int s = 0; s < PSUB; ++s) tma_load_3d(sX + s * SSD_SUB, &tmX, b_tma, s * 64, c0, h);
      if (ch + 1 < ch1) {   // the coming chunk's tiles start on their way to L2
        for (int s = 0; s < nsub; ++s) {
          if (!LOCAL) tma_prefetch_3d(&tmBC, s * 64, c0 + 128, L.groups + grp);
          tma_prefetch_3d(&tmBC, s * 64, c0 + 128, grp);
        }
        for (int s = 0; s < PSUB; ++s) tma_prefetch_3d(&tmX, s * 64, c0 + 128, h);
      }
    }
    __syncwarp();
    const float d = d_next;
    float cum = cum_next;
    for (int w = 0; w < (warp & 3); ++w) cum += s_part[half * 4 + w];
    const float total = (s_part[0] + s_part[1]) + (s_part[2] + s_part[3]);
    load_dt(ch + 1);
    decay_log += total;
    if (half == 0) s_e[row] = d > 0.f ? cum - log2f(d) : INFINITY;   // W_ij = G_ij 2^(cum_i - e_j)
    // the state as an operand (two terms), and scaled for the accumulation that follows
    {
      const float dec = exp2f(total);
#pragma unroll
      for (int c = 0; c < HC; c += 32) {
        uint32_t r[32];
        float v[32];
        tmem_ld32(tS + c, r);
        if (ch > ch0) {
          uint32_t t[32];
          tmem_ld32(tT + c, t);
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]) + __uint_as_float(t[j]);
        } else {
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]);
        }
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          r[j] = __float_as_uint(v[j] * dec);
        }
        tmem_st32(tS + c, r);
        if (!LOCAL) store_split(sS, sSl, row, half * HC + c, v);
      }
      tmem_wait_st();
    }
    fence_proxy_async_smem();
    tc_fence_before();
    ok = mbar_wait(b_tma, ph);
    ok = __syncthreads_and(ok);
    if (!ok) {
      if (threadIdx.x == 0) set_error(err, ERR_WAIT_MMA_FULL);
      break;
    }
    if constexpr (!LOCAL) {
    if (threadIdx.x == 0) {
      tc_fence_after();
      constexpr uint32_t id_g = umma_idesc(1, 1, 1, 0, 0, 128, 128), id_y = umma_idesc(1, 1, 1, 0, 1, 128, PP);
      const uint32_t aC = smem_u32(sC), aB = smem_u32(sB), aS = smem_u32(sS), aSl = smem_u32(sSl);
      for (int t = 0; t < nk; ++t) {
        const uint32_t o = (t / 4) * SSD_SUB + (t % 4) * 32;
        umma_f16_ss(tm + Cfg::COL_G, umma_smem_desc(aC + o, 16, 1024), umma_smem_desc(aB + o, 16, 1024), id_g, t != 0);
      }
      for (int t = 0; t < nk; ++t) {
        const uint32_t o = (t / 4) * SSD_SUB + (t % 4) * 32;
        umma_f16_ss(tm + Cfg::COL_Y, umma_smem_desc(aC + o, 16, 1024), umma_smem_desc(aS + t * 2048, SSD_SUB, 1024), id_y,
                    t != 0);
        umma_f16_ss(tm + Cfg::COL_Y, umma_smem_desc(aC + o, 16, 1024), umma_smem_desc(aSl + t * 2048, SSD_SUB, 1024), id_y, 1);
      }
      umma_commit(b_gy);
    }
    __syncwarp();
    ok = mbar_wait(b_gy, ph);
    tc_fence_after();
    __syncwarp();
    // scores of this thread's 64 columns into registers before any thread writes weights over them
    uint32_t g0[32], g1[32];
    tmem_ld32(tG + half * 64, g0);
    tmem_ld32(tG + half * 64 + 32, g1);
    tmem_wait_ld();
    tc_fence_before();
    ok = __syncthreads_and(ok);
    if (!ok) {
      if (threadIdx.x == 0) set_error(err, ERR_WAIT_EPILOGUE);
      break;
    }
    tc_fence_after();
    {
      const float* e = s_e + half * 64;
      const int lim = row - half * 64;   // columns j <= lim are in the past
      auto weights = [&](const uint32_t (&g)[32], int j0) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int j = 0; j < 32; j += 4) {
          const float4 ev = *reinterpret_cast<const float4*>(e + j0 + j);
          const float w0 = j0 + j <= lim ? __uint_as_float(g[j]) * exp2f(cum - ev.x) : 0.f;
          const float w1 = j0 + j + 1 <= lim ? __uint_as_float(g[j + 1]) * exp2f(cum - ev.y) : 0.f;
          const float w2 = j0 + j + 2 <= lim ? __uint_as_float(g[j + 2]) * exp2f(cum - ev.z) : 0.f;
          const float w3 = j0 + j + 3 <= lim ? __uint_as_float(g[j + 3]) * exp2f(cum - ev.w) : 0.f;
          const float2 s01 = split_pair(w0, w1), s23 = split_pair(w2, w3);
          hi[j >> 1] = __float_as_uint(s01.x);
          lo[j >> 1] = __float_as_uint(s01.y);
          hi[(j >> 1) + 1] = __float_as_uint(s23.x);
          lo[(j >> 1) + 1] = __float_as_uint(s23.y);
        }
        tmem_st16(tG + half * 32 + (j0 >> 1), hi);
        tmem_st16(tG + 64 + half * 32 + (j0 >> 1), lo);
      };
      weights(g0, 0);
      weights(g1, 32);
    }
    }
    {
      const float sc = exp2f(cum), w = d * exp2f(total - cum);
#pragma unroll
      for (int c = 0; c < HC; c += 32) {
        if constexpr (!LOCAL) {
          uint32_t r[32];
          tmem_ld32(tY + c, r);
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * sc);
          tmem_st32(tY + c, r);
        }
        float v[32];
        const int col0 = half * HC + c;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int col = col0 + q * 8;
          float f[8];
          unpack8(*reinterpret_cast<const bf16x8*>(sX + (col >> 6) * SSD_SUB + row * 128 +
                                                   ((((col & 63) >> 3) ^ (row & 7)) << 4)), f);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[q * 8 + j] = f[j] * w;
        }
        store_split(sS, sSl, row, col0, v);   // the state operand is behind its products
      }
    }
    tmem_wait_st();
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0) {
      tc_fence_after();
      constexpr uint32_t id_y = umma_idesc(1, 1, 1, 0, 1, 128, PP), id_s = umma_idesc(1, 1, 1, 1, 1, 128, PP),
                         id_s2 = umma_idesc(1, 1, 1, 1, 1, 128, 2 * PP);
      const uint32_t aB = smem_u32(sB), aX = smem_u32(sX), aW = smem_u32(sS), aWl = smem_u32(sSl);
#pragma unroll
      for (int t = 0; t < (LOCAL ? 0 : 8); ++t) {
        umma_f16_ts(tm + Cfg::COL_Y, tm + Cfg::COL_G + t * 8, umma_smem_desc(aX + t * 2048, SSD_SUB, 1024), id_y, 1);
        umma_f16_ts(tm + Cfg::COL_Y, tm + Cfg::COL_G + 64 + t * 8, umma_smem_desc(aX + t * 2048, SSD_SUB, 1024), id_y, 1);
      }
      if (!LOCAL) umma_commit(b_y);
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        const uint64_t da = umma_smem_desc(aB + t * 2048, SSD_SUB, 1024);
        if (t == 0) {   // S goes on, T starts anew
          umma_f16_ss(tm + Cfg::COL_S, da, umma_smem_desc(aW, SSD_SUB, 1024), id_s, 1);
          umma_f16_ss(tm + Cfg::COL_T, da, umma_smem_desc(aWl, SSD_SUB, 1024), id_s, 0);
        } else {
          umma_f16_ss(tm + Cfg::COL_S, da, umma_smem_desc(aW + t * 2048, SSD_SUB, 1024), id_s2, 1);
        }
      }
      umma_commit(b_s);
    }
    __syncwarp();
    if constexpr (!LOCAL) {
    ok = mbar_wait(b_y, ph);
    tc_fence_after();
    __syncwarp();
    // outputs go through the C tile's place (its products are behind us), so that a row's columns leave
    // as one contiguous piece
#pragma unroll
    for (int c = 0; c < HC; c += 32) {
      uint32_t r[32];
      tmem_ld32(tY + c, r);
      tmem_wait_ld();
      const int col0 = half * HC + c;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int col = col0 + q * 8;
        float f[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sX + (col >> 6) * SSD_SUB + row * 128 +
                                                 ((((col & 63) >> 3) ^ (row & 7)) << 4)), f);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = fmaf(D, f[j], __uint_as_float(r[q * 8 + j]));
        store8(reinterpret_cast<__nv_bfloat16*>(sC + (col >> 6) * SSD_SUB + row * 128 +
                                                ((((col & 63) >> 3) ^ (row & 7)) << 4)), f);
      }
    }
    ok = __syncthreads_and(ok);
    if (ok) {
      constexpr int VR = PP / 8;   // 16-byte pieces of a row
      for (int i = threadIdx.x; i < valid * VR; i += SSD_THREADS) {
        const int rr = i / VR, q = i % VR;
        if (q * 8 < L.p)
          *reinterpret_cast<uint4*>(y + (size_t)(c0 + rr) * ldy + h * L.p + q * 8) =
              *reinterpret_cast<const uint4*>(sC + (q >> 3) * SSD_SUB + rr * 128 + (((q & 7) ^ (rr & 7)) << 4));
      }
    }
    }
    scan_dt();
    fence_proxy_async_smem();     // the C tile's place was read and written by threads; TMA writes it next
    ok = mbar_wait(b_s, ph) && ok;
    tc_fence_after();
    ok = __syncthreads_and(ok);   // every tile and the accumulators are free for the next chunk
    if (!ok && threadIdx.x == 0) set_error(err, ERR_WAIT_EPILOGUE);
  }
  __syncwarp();
  if (LOCAL && threadIdx.x == 0) s_dec[z] = exp2f(decay_log);
  if (ok && ch1 > ch0 && (LOCAL || z == z_last)) {
    float* dst = LOCAL ? sg + z * np : state;
#pragma unroll
    for (int c = 0; c < HC; c += 32) {
      uint32_t r[32], t[32];
      tmem_ld32(tS + c, r);
      tmem_ld32(tT + c, t);
      tmem_wait_ld();
#pragma unroll
      for (int j = 0; j < 32; ++j)
        s_st[row * PP + ((half * HC + c + j) ^ (row & 31))] = __uint_as_float(r[j]) + __uint_as_float(t[j]);
    }
    __syncthreads();
#pragma unroll 4
    for (int n = warp; n < L.n; n += SSD_THREADS / 32) {
#pragma unroll
      for (int p0 = 0; p0 < PP; p0 += 32) {
        const int p = p0 + lane;
        if (p < L.p) dst[(size_t)n * L.p + p] = s_st[n * PP + (p ^ (n & 31))];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tm, Cfg::TMEM_COLS);
  }
}

template <int PP>
static int launch_ssd(const CUtensorMap& tmBC, const CUtensorMap& tmX, const BbHyLayer& L, const BbHyWork& w,
                      const BbHyBatch& b, cudaStream_t s) {
  static PerDeviceOnce once, once_local;
  constexpr int SMEM = SsdCfg<PP>::SMEM;
  cudaError_t e = ensure_dyn_smem(once, ssd_chunk_kernel<PP, false>, SMEM);
  if (e != cudaSuccess) return (int)e;
  e = ensure_dyn_smem(once_local, ssd_chunk_kernel<PP, true>, SMEM);
  if (e != cudaSuccess) return (int)e;
  // segments: as many as fill the machine once, of four chunks or more (a 2048-token prompt of 64 heads
  // alone: 75 us against 112 us in one piece; at two chunks the extra launch costs more than it saves),
  // and as the scratch allows
  const long pairs = (long)b.ns_pre * L.heads, np = (long)L.n * L.p;
  int segs = (int)((PP == 64 ? 2 : 1) * sm_count() / pairs);
  const int most = (b.max_len + 127) / 128 / 4;
  if (segs > most) segs = most;
  if (segs > 16) segs = 16;
  while (segs > 1 && pairs * ((segs + 1) * np + segs) > w.seg_floats) --segs;
  if (segs < 2) segs = 1;
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(w.y);
  const dim3 grid(b.ns_pre, L.heads, segs);
  if (segs > 1) {
    ssd_chunk_kernel<PP, true><<<grid, SSD_THREADS, SMEM, s>>>(tmBC, tmX, L, w.dt, w.ld_dt, y, w.ld_y, b, segs, w.seg,
                                                               device_error_word());
    e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
  }
  ssd_chunk_kernel<PP, false><<<grid, SSD_THREADS, SMEM, s>>>(tmBC, tmX, L, w.dt, w.ld_dt, y, w.ld_y, b, segs, w.seg,
                                                              device_error_word());
  return (int)cudaGetLastError();
}

}  // namespace bb

// Prompt portions of one layer, bf16; BB_ESIZE for sizes it does not cover (the caller then runs the
// token-by-token scan): head and state sizes are multiples of 8 up to 128.
BB_API int bb_ssd_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  using namespace bb;
  if (b->ns_pre <= 0) return BB_OK;
  if (c->dtype || L->n % 8 || L->p % 8 || L->n > 128 || L->p > 128) return BB_ESIZE;
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(w->xbc);
  const uint64_t ld = (uint64_t)w->ld_xbc * 2;
  CUtensorMap tmBC, tmX;
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&tmBC, bf, 2, xbc + L->inner, L->n, b->n_pre, 2 * L->groups, ld, (uint64_t)L->n * 2, 64, 128);
  if (rc) return rc;
  rc = make_tmap_3d(&tmX, bf, 2, xbc, L->p, b->n_pre, L->heads, ld, (uint64_t)L->p * 2, 64, 128);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return L->p <= 64 ? launch_ssd<64>(tmBC, tmX, *L, *w, *b, s) : launch_ssd<128>(tmBC, tmX, *L, *w, *b, s);
}

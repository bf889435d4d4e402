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
// GATED: the same chunks for a matrix memory with exponential gates (mLSTM), C, B, X being its queries, keys and
// values.  With F the running sum of the log forget gates inside the chunk, e = i - F and M_i the running maximum of
// (m before the chunk, e), the stabiliser is m_i = F_i + M_i and every exponent below is at most 0:
//   W_ij = G_ij exp(e_j - M_i),   Y = exp(m - M_i) (C S) + W X,   S = exp(m - M_last) S + B^T (exp(e_j - M_last) x_j)
// The normaliser n follows S (in shared memory, on the CUDA cores): n.q_i is exp(m - M_i) (n.q_i) plus the sum of
// row i of W.  A row leaves divided by max(|n.q|, exp(-m_i)), over its root mean square, times gain and gate.
//
// Without step sizes (dt null) they are 1 and the outputs take the factor q_scale: retention, whose decays are constants
// of the heads.
//
// With few (sequence, head) pairs a portion is cut into segments of whole chunks that run side by side:
// a first launch (LOCAL) computes what each segment adds to the state on its own, and its decay; the
// segments of the main launch then start from the state carried in, decayed and summed over the segments
// before them (GATED: each brought to a common stabiliser).
//
// TMEM lane = token (or state row); W warpgroups share a row's columns: two, or four where one CTA has the SM to
// itself and GATED has the most to do between the MMAs.  Thread 0 issues TMA and MMA.  The phases of a chunk
// are separated by block barriers; with head sizes up to 64 two CTAs share an SM (113 KB of shared memory, 256
// TMEM columns each) and fill each other's gaps.
// TMEM: G, then W as packed bf16 (value in its first 64 columns, remainder in the others); Y; S.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../common/split.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

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
  static constexpr int W = 2, GATED_W = PP == 64 ? 2 : 4;       // warpgroups
  static constexpr int GATED_FLOATS = 128 * (2 + 6 * GATED_W) + 64;   // see GatedSmem
  // TMEM columns.  The state product of a chunk leaves its two terms side by side: the first added to S,
  // the second in T right behind it (one 2 PP wide MMA per step instead of two, which cost the same each).
  // With PP = 64 T lies over the first half of W, whose products are issued before.
  static constexpr int COL_G = PP == 64 ? 128 : 0, COL_Y = PP == 64 ? 0 : 128, COL_S = PP == 64 ? 64 : 256;
  static constexpr int COL_T = COL_S + PP;
  static constexpr int TMEM_COLS = PP == 64 ? 256 : 512;
};

// What the gated form keeps beside the tiles: with head sizes up to 64 in the half of the query tile that stays free
// (two CTAs then still share an SM), else behind everything.
template <int W>
struct GatedSmem {
  float *n, *w, *sum, *nq, *part, *pm, *co;   // [128] normaliser, [128] token weights, [W][128] sums of a row's parts,
                                              // [W][128] n.q likewise, [4 W][128], [4], [34]
  __device__ explicit GatedSmem(float* p)
      : n(p), w(p + 128), sum(p + 256), nq(sum + W * 128), part(nq + W * 128), pm(part + 4 * W * 128), co(pm + 4) {}
};

template <int PP, bool LOCAL, bool GATED, int W>
__global__ void __launch_bounds__(W * 128, PP == 64 ? 2 : 1)
ssd_chunk_kernel(const __grid_constant__ CUtensorMap tmBC, const __grid_constant__ CUtensorMap tmX,
                 const __grid_constant__ BbHyLayer L, const float* __restrict__ dt, int lddt,
                 __nv_bfloat16* __restrict__ y, int ldy, const __grid_constant__ BbHyBatch b, int segs,
                 float* __restrict__ seg, int* err, const __nv_bfloat16* __restrict__ proj, int ldp, float eps) {
  using Cfg = SsdCfg<PP>;
  constexpr int SSD_THREADS = W * 128;
  constexpr int PSUB = Cfg::PSUB, HC = PP / W, GC = 128 / W;   // Y / S / X columns and G columns of a thread
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sC = smem + Cfg::OFF_C;
  uint8_t* sB = smem + Cfg::OFF_B;
  uint8_t* sX = smem + Cfg::OFF_X;
  uint8_t* sS = smem + Cfg::OFF_S;
  uint8_t* sSl = sS + PSUB * SSD_SUB;
  float* s_e = reinterpret_cast<float*>(smem + Cfg::OFF_E);   // [128]
  float* s_part = s_e + 128;                                  // [4] (of 8) warp sums of the coming chunk
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
  const float a2 = GATED ? 0.f : L.a[h] * kLog2e, D = GATED || !L.d_skip ? 0.f : L.d_skip[h];
  const float y_scale = GATED || dt ? 1.f : L.q_scale;
  const int pw = GATED || !L.pp ? L.p : L.pp;                   // columns of a head in the output
  const size_t np = (size_t)L.n * L.p, mem = GATED ? L.mem : np;   // floats of a state
  float* state = L.ssm_state + ((size_t)slot * L.heads + h) * mem;
  GatedSmem<W> gs(reinterpret_cast<float*>(PP == 64 && nsub == 1 ? sC + SSD_SUB : smem + Cfg::SMEM));

  // this CTA's chunks, and the scratch of its (sequence, head): segment states, the state carried in, decays
  const int z = blockIdx.z, per = (n_chunks + segs - 1) / segs, z_last = (n_chunks - 1) / per;
  if (z > z_last || (LOCAL && z > 0 && z == z_last)) return;
  const int ch0 = z * per, ch1 = LOCAL && z == z_last ? ch0 : min(n_chunks, ch0 + per);
  float* sg = seg + ((size_t)seq * L.heads + h) * ((segs + 1) * mem + segs);
  float* s_carry = sg + segs * mem;
  float* s_dec = s_carry + mem;                                  // GATED: sum of the log forget gates

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
  const uint32_t tG = tm + Cfg::COL_G + lane_sel, tY = tm + Cfg::COL_Y + lane_sel + half * HC,
                 tS = tm + Cfg::COL_S + lane_sel + half * HC, tT = tm + Cfg::COL_T + lane_sel + half * HC;
  // The state between memory and TMEM goes through the operand tiles' place as fp32 [128][PP], columns
  // exclusive-or'ed with the row: a warp moves whole rows of memory, a thread reads or writes its own row.
  float* s_st = reinterpret_cast<float*>(sS);
  {
    const bool fresh = b.seq_pos0[seq] == 0;
    if constexpr (GATED) {
      // the normaliser and the stabiliser (log2 units) this CTA starts from; factors of the segments before it
      if (threadIdx.x == 0) {
        float m = -INFINITY;
        if (LOCAL ? z == 0 : segs == 1) m = fresh ? 0.f : state[np + L.n] * kLog2e;
        else if (!LOCAL) m = z == 0 ? s_carry[np + L.n] : sg[np + L.n];
        for (int k = 1; !LOCAL && k < z; ++k) {
          const float own = sg[k * mem + np + L.n], next = fmaxf(m + s_dec[k], own);
          gs.co[2 * k] = exp2f(m + s_dec[k] - next);
          gs.co[2 * k + 1] = exp2f(own - next);
          m = next;
        }
        gs.co[0] = m;
        if (LOCAL && z == 0) s_carry[np + L.n] = m;
      }
      __syncthreads();
      if (threadIdx.x < 128) {
        const int d = threadIdx.x;
        float v = 0.f;
        if (d < L.n) {
          if (LOCAL ? z == 0 : segs == 1) v = fresh ? 0.f : state[np + d];
          else if (!LOCAL) v = z == 0 ? s_carry[np + d] : sg[np + d];
          if (LOCAL && z == 0) s_carry[np + d] = v;
          for (int k = 1; !LOCAL && k < z; ++k) v = v * gs.co[2 * k] + sg[k * mem + np + d] * gs.co[2 * k + 1];
        }
        gs.n[d] = v;
      }
    }
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
            for (int k = 1; k < z; ++k) {
              if constexpr (GATED) v = v * gs.co[2 * k] + sg[k * mem + i] * gs.co[2 * k + 1];
              else v = fmaf(v, s_dec[k], sg[k * mem + i]);
            }
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
  // (GATED: log input gate in d_next, log forget gate and its sum in cum_next, running maximum of e in max_next)
  float d_next = 0.f, cum_next = 0.f, max_next = 0.f;
  auto load_dt = [&](int ch) {
    const int i = ch * 128 + row;
    if constexpr (GATED) {
      d_next = i < len ? dt[(size_t)(r0 + i) * lddt + L.off32_i + h] * kLog2e : -INFINITY;
      cum_next = i < len ? dt[(size_t)(r0 + i) * lddt + L.off32_f + h] * kLog2e : 0.f;
    } else {
      d_next = i < len ? (dt ? dt[(size_t)(r0 + i) * lddt + h] : 1.f) : 0.f;
    }
  };
  auto scan_dt = [&]() {
    if (!GATED) cum_next = a2 * d_next;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, cum_next, o);
      if (lane >= o) cum_next += v;
    }
    if (lane == 31 && half == 0) s_part[warp] = cum_next;
    if constexpr (GATED) {
      d_next -= cum_next;                          // e, less the sum over the warps before this one
      max_next = d_next;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, max_next, o);
        if (lane >= o) max_next = fmaxf(max_next, v);
      }
      if (lane == 31 && half == 0) gs.pm[warp] = max_next;
    }
  };
  load_dt(ch0);
  scan_dt();
  __syncthreads();

  bool ok = (smem_u32(smem) & 1023u) == 0;
  if (!ok && threadIdx.x == 0) set_error(err, ERR_BAD_ARG);
  float decay_log = 0.f;
  float m_run = GATED ? gs.co[0] : 0.f;
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
    const float total = (s_part[0] + s_part[1]) + (s_part[2] + s_part[3]);
    // of this row: W_ij = G_ij 2^(w_row - s_e[j]), factor on what the state adds, factor as an input of the state;
    // of the chunk: factor on the state.  GATED: log2 of the stabiliser as well
    float w_row, sc, w_in, dec, m_row = 0.f;
    if constexpr (GATED) {
      float base = 0.f, mine = 0.f, top = m_run, top_all = m_run;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        if (w == (warp & 3)) {
          mine = base;
          top = top_all;
        }
        top_all = fmaxf(top_all, gs.pm[w] - base);
        base += s_part[w];
      }
      const float e = d - mine;
      top = fmaxf(top, max_next - mine);
      m_row = mine + cum_next + top;
      w_row = -top;
      sc = exp2f(m_run - top);
      w_in = exp2f(e - top_all);
      dec = exp2f(m_run - top_all);
      m_run = total + top_all;
      if (half == 0) {
        s_e[row] = -e;
        gs.w[row] = w_in;
      }
    } else {
      float cum = cum_next;
      for (int w = 0; w < (warp & 3); ++w) cum += s_part[w];
      w_row = cum;
      dec = exp2f(total);
      if (half == 0) s_e[row] = d > 0.f ? cum - log2f(d) : INFINITY;
    }
    load_dt(ch + 1);
    decay_log += total;
    // the state as an operand (two terms), and scaled for the accumulation that follows
    {
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
        if (!LOCAL) store_split(sS, sSl, row, half * HC + c, v, SSD_SUB);
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
    if constexpr (GATED) {
      // this row's query with the normaliser, a part of the channels to a thread
      const int vecs = nsub * 8 / W, vec0 = half * vecs;      // vectors of 8 channels
      float a = 0.f;
      for (int v = 0; v < vecs; ++v) {
        const int q = vec0 + v;
        float f[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sC + (q >> 3) * SSD_SUB + row * 128 + (((q & 7) ^ (row & 7)) << 4)), f);
        const float4 n0 = *reinterpret_cast<const float4*>(gs.n + q * 8), n1 = *reinterpret_cast<const float4*>(gs.n + q * 8 + 4);
        a = fmaf(f[0], n0.x, fmaf(f[1], n0.y, fmaf(f[2], n0.z, fmaf(f[3], n0.w, a))));
        a = fmaf(f[4], n1.x, fmaf(f[5], n1.y, fmaf(f[6], n1.z, fmaf(f[7], n1.w, a))));
      }
      gs.nq[half * 128 + row] = a * sc;
    }
    ok = mbar_wait(b_gy, ph);
    tc_fence_after();
    __syncwarp();
    // scores of this thread's columns into registers before any thread writes weights over them
    uint32_t g0[32], g1[GC == 64 ? 32 : 1];
    tmem_ld32(tG + half * GC, g0);
    if constexpr (GC == 64) tmem_ld32(tG + half * GC + 32, g1);
    tmem_wait_ld();
    tc_fence_before();
    ok = __syncthreads_and(ok);
    if (!ok) {
      if (threadIdx.x == 0) set_error(err, ERR_WAIT_EPILOGUE);
      break;
    }
    tc_fence_after();
    {
      const float* e = s_e + half * GC;
      const int lim = row - half * GC;   // columns j <= lim are in the past
      float row_sum = 0.f;
      auto weights = [&](const uint32_t (&g)[32], int j0) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int j = 0; j < 32; j += 4) {
          const float4 ev = *reinterpret_cast<const float4*>(e + j0 + j);
          const float w0 = j0 + j <= lim ? __uint_as_float(g[j]) * exp2f(w_row - ev.x) : 0.f;
          const float w1 = j0 + j + 1 <= lim ? __uint_as_float(g[j + 1]) * exp2f(w_row - ev.y) : 0.f;
          const float w2 = j0 + j + 2 <= lim ? __uint_as_float(g[j + 2]) * exp2f(w_row - ev.z) : 0.f;
          const float w3 = j0 + j + 3 <= lim ? __uint_as_float(g[j + 3]) * exp2f(w_row - ev.w) : 0.f;
          if (GATED) row_sum += (w0 + w1) + (w2 + w3);
          const float2 s01 = split_pair(w0, w1), s23 = split_pair(w2, w3);
          hi[j >> 1] = __float_as_uint(s01.x);
          lo[j >> 1] = __float_as_uint(s01.y);
          hi[(j >> 1) + 1] = __float_as_uint(s23.x);
          lo[(j >> 1) + 1] = __float_as_uint(s23.y);
        }
        tmem_st16(tG + half * (GC / 2) + (j0 >> 1), hi);
        tmem_st16(tG + 64 + half * (GC / 2) + (j0 >> 1), lo);
      };
      weights(g0, 0);
      if constexpr (GC == 64) weights(g1, 32);
      if (GATED) gs.sum[half * 128 + row] = row_sum;
    }
    }
    {
      if constexpr (!GATED) {
        sc = exp2f(w_row);
        w_in = d * exp2f(total - w_row);
      }
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
          for (int j = 0; j < 8; ++j) v[q * 8 + j] = f[j] * w_in;
        }
        store_split(sS, sSl, row, col0, v, SSD_SUB);   // the state operand is behind its products
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
    if constexpr (GATED) {
      // the normaliser's new part: 8 channels of a few tokens to a thread, summed over the CTA below
      const int nv = nsub * 8, v = threadIdx.x % nv, per = nv / W, t0 = threadIdx.x / nv * per;
      float a[8] = {};
#pragma unroll 4
      for (int t = t0; t < t0 + per; ++t) {
        float f[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sB + (v >> 3) * SSD_SUB + t * 128 + (((v & 7) ^ (t & 7)) << 4)), f);
        const float w = gs.w[t];
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] = fmaf(w, f[j], a[j]);
      }
      for (int o = nv; o < 32; o <<= 1)
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] += __shfl_xor_sync(0xffffffffu, a[j], o);
      if (lane < nv) {
        float4* p = reinterpret_cast<float4*>(gs.part + warp * 128 + v * 8);
        p[0] = make_float4(a[0], a[1], a[2], a[3]);
        p[1] = make_float4(a[4], a[5], a[6], a[7]);
      }
    }
    if constexpr (!LOCAL) {
    ok = mbar_wait(b_y, ph);
    tc_fence_after();
    __syncwarp();
    // outputs go through the C tile's place (its products are behind us), so that a row's columns leave
    // as one contiguous piece
    if constexpr (GATED) {
      float nq = 0.f;
#pragma unroll
      for (int w = 0; w < W; ++w) nq += gs.nq[w * 128 + row] + gs.sum[w * 128 + row];
      nq *= L.q_scale;
      const float f = L.q_scale / (fmaxf(fabsf(nq), exp2f(-m_row)) + 1e-6f);
      float o[HC], ss = 0.f;
#pragma unroll
      for (int c = 0; c < HC; c += 32) {
        uint32_t r[32];
        tmem_ld32(tY + c, r);
        tmem_wait_ld();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          o[c + j] = __uint_as_float(r[j]) * f;
          ss = fmaf(o[c + j], o[c + j], ss);
        }
      }
      // (the row's sums have been read by both of its threads when the barrier is behind them)
      ok = __syncthreads_and(ok);
      gs.sum[half * 128 + row] = ss;
      if (threadIdx.x < L.n) {
        float v = gs.n[threadIdx.x] * dec;
#pragma unroll
        for (int w = 0; w < 4 * W; ++w) v += gs.part[w * 128 + threadIdx.x];
        gs.n[threadIdx.x] = v;
      }
      __syncthreads();
      ss = 0.f;
#pragma unroll
      for (int w = 0; w < W; ++w) ss += gs.sum[w * 128 + row];
      const float rstd = rsqrtf(ss / (float)L.p + eps);
#pragma unroll
      for (int q = 0; q < HC / 8; ++q) {
        const int col = half * HC + q * 8;
        float x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = o[q * 8 + j] * rstd;
        store8(reinterpret_cast<__nv_bfloat16*>(sC + (col >> 6) * SSD_SUB + row * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4)), x);
      }
    } else {
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
        for (int j = 0; j < 8; ++j) f[j] = fmaf(D, f[j], __uint_as_float(r[q * 8 + j]) * y_scale);
        store8(reinterpret_cast<__nv_bfloat16*>(sC + (col >> 6) * SSD_SUB + row * 128 +
                                                ((((col & 63) >> 3) ^ (row & 7)) << 4)), f);
      }
    }
    }
    constexpr int VR = PP / 8;     // 16-byte pieces of a row
    constexpr int OUT_IT = 128 * VR / SSD_THREADS;
    bf16x8 gate[GATED ? OUT_IT : 1];
    if constexpr (GATED) {         // output gates, asked for ahead of the barrier
#pragma unroll
      for (int it = 0; it < OUT_IT; ++it) {
        const int i = threadIdx.x + it * SSD_THREADS, rr = i / VR, q = i % VR;
        if (rr < valid && q * 8 < L.pp)
          gate[it] = *reinterpret_cast<const bf16x8*>(proj + (size_t)(c0 + rr) * ldp + L.off_gg + h * L.pp + q * 8);
      }
    }
    ok = __syncthreads_and(ok);
    if constexpr (GATED) {
#pragma unroll
      for (int it = 0; it < OUT_IT; ++it) {
        const int i = threadIdx.x + it * SSD_THREADS, rr = i / VR, q = i % VR, col = h * L.pp + q * 8;
        if (ok && rr < valid && q * 8 < L.pp) {
          float f[8], g[8], w[8];
          unpack8(*reinterpret_cast<const bf16x8*>(sC + (q >> 3) * SSD_SUB + rr * 128 + (((q & 7) ^ (rr & 7)) << 4)), f);
          unpack8(gate[it], g);
          load8(L.gnorm + col, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] *= w[j] * sigmoid_as<__nv_bfloat16>(g[j]);
          store8(y + (size_t)(c0 + rr) * ldy + col, f);
        }
      }
    } else if (ok) {
      for (int i = threadIdx.x; i < valid * VR; i += SSD_THREADS) {
        const int rr = i / VR, q = i % VR;
        if (q * 8 < pw)
          *reinterpret_cast<uint4*>(y + (size_t)(c0 + rr) * ldy + h * pw + q * 8) =
              *reinterpret_cast<const uint4*>(sC + (q >> 3) * SSD_SUB + rr * 128 + (((q & 7) ^ (rr & 7)) << 4));
      }
    }
    } else if constexpr (GATED) {
      __syncthreads();
      if (threadIdx.x < L.n) {
        float v = gs.n[threadIdx.x] * dec;
#pragma unroll
        for (int w = 0; w < 4 * W; ++w) v += gs.part[w * 128 + threadIdx.x];
        gs.n[threadIdx.x] = v;
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
  if (LOCAL && threadIdx.x == 0) s_dec[z] = GATED ? decay_log : exp2f(decay_log);
  if (ok && ch1 > ch0 && (LOCAL || z == z_last)) {
    float* dst = LOCAL ? sg + z * mem : state;
    if constexpr (GATED) {       // the stabiliser in log2 units between the segments, else in natural ones
      if (threadIdx.x < L.n) dst[np + threadIdx.x] = gs.n[threadIdx.x];
      if (threadIdx.x == 0) dst[np + L.n] = LOCAL ? m_run : m_run * 0.69314718055994531f;
    }
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

// y: outputs of the recurrence, or with GATED the finished rows of the mixer; dt: step sizes, or log gates.
template <int PP, bool GATED>
static int launch_ssd(const CUtensorMap& tmBC, const CUtensorMap& tmX, const BbHyLayer& L, const BbHyWork& w,
                      const BbHyBatch& b, const float* dt, int lddt, __nv_bfloat16* y, int ldy, float eps, cudaStream_t s) {
  static PerDeviceOnce once, once_local;
  constexpr int W = GATED ? SsdCfg<PP>::GATED_W : SsdCfg<PP>::W;
  constexpr int MOST = SsdCfg<PP>::SMEM + (GATED ? 4 * SsdCfg<PP>::GATED_FLOATS : 0);
  cudaError_t e = ensure_dyn_smem(once, ssd_chunk_kernel<PP, false, GATED, W>, MOST);
  if (e != cudaSuccess) return (int)e;
  e = ensure_dyn_smem(once_local, ssd_chunk_kernel<PP, true, GATED, W>, MOST);
  if (e != cudaSuccess) return (int)e;
  const int smem = GATED && (PP > 64 || L.n > 64) ? MOST : SsdCfg<PP>::SMEM;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(w.proj);
  // segments: as many as fill the machine once, of four chunks or more (a 2048-token prompt of 64 heads
  // alone: 75 us against 112 us in one piece; at two chunks the extra launch costs more than it saves; GATED: of two),
  // and as the scratch allows
  const long pairs = (long)b.ns_pre * L.heads, np = GATED ? L.mem : (long)L.n * L.p;
  int segs = (int)((PP == 64 && smem < 116 * 1024 ? 2 : 1) * sm_count() / pairs);
  const int most = (b.max_len + 127) / 128 / (GATED ? 2 : 4);
  if (segs > most) segs = most;
  if (segs > 16) segs = 16;
  while (segs > 1 && pairs * ((segs + 1) * np + segs) > w.seg_floats) --segs;
  if (segs < 2) segs = 1;
  const dim3 grid(b.ns_pre, L.heads, segs);
  if (segs > 1) {
    ssd_chunk_kernel<PP, true, GATED, W><<<grid, W * 128, smem, s>>>(tmBC, tmX, L, dt, lddt, y, ldy, b, segs, w.seg,
                                                                      device_error_word(), proj, w.ld_proj, eps);
    e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
  }
  ssd_chunk_kernel<PP, false, GATED, W><<<grid, W * 128, smem, s>>>(tmBC, tmX, L, dt, lddt, y, ldy, b, segs, w.seg,
                                                                     device_error_word(), proj, w.ld_proj, eps);
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
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(w->y);
  return L->p <= 64 ? launch_ssd<64, false>(tmBC, tmX, *L, *w, *b, w->dt, w->ld_dt, y, w->ld_y, 0.f, s)
                    : launch_ssd<128, false>(tmBC, tmX, *L, *w, *b, w->dt, w->ld_dt, y, w->ld_y, 0.f, s);
}

// The same for a matrix memory, from log gates in w->f32: recurrence, norm and gate -> w->cat.  BB_ESIZE for heads
// above 128.
BB_API int bb_mlstm_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  using namespace bb;
  if (b->ns_pre <= 0) return BB_OK;
  if (c->dtype || L->np > 128 || L->pp > 128) return BB_ESIZE;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(w->proj);
  const uint64_t ld = (uint64_t)w->ld_proj * 2;
  CUtensorMap tmBC, tmX;
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&tmBC, bf, 2, proj + L->off_kk, L->np, b->n_pre, 2 * L->heads, ld, (uint64_t)L->np * 2, 64, 128);
  if (rc) return rc;
  rc = make_tmap_3d(&tmX, bf, 2, proj + L->off_vv, L->pp, b->n_pre, L->heads, ld, (uint64_t)L->pp * 2, 64, 128);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  __nv_bfloat16* cat = static_cast<__nv_bfloat16*>(w->cat);
  return L->p <= 64 ? launch_ssd<64, true>(tmBC, tmX, *L, *w, *b, w->f32, w->ld_f32, cat, w->ld_cat, c->eps, s)
                    : launch_ssd<128, true>(tmBC, tmX, *L, *w, *b, w->f32, w->ld_f32, cat, w->ld_cat, c->eps, s);
}

// The same for retention: queries and keys (rotated) and values in w->proj -> outputs in w->y.  BB_ESIZE for heads above 128.
BB_API int bb_retention_chunk(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, void* stream) {
  using namespace bb;
  if (b->ns_pre <= 0) return BB_OK;
  if (c->dtype || L->np > 128 || L->pp > 128) return BB_ESIZE;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(w->proj);
  const uint64_t ld = (uint64_t)w->ld_proj * 2;
  CUtensorMap tmBC, tmX;
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&tmBC, bf, 2, proj + L->off_kk, L->np, b->n_pre, 2 * L->heads, ld, (uint64_t)L->np * 2, 64, 128);
  if (rc) return rc;
  rc = make_tmap_3d(&tmX, bf, 2, proj + L->off_vv, L->pp, b->n_pre, L->heads, ld, (uint64_t)L->pp * 2, 64, 128);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(w->y);
  return L->p <= 64 ? launch_ssd<64, false>(tmBC, tmX, *L, *w, *b, nullptr, 0, y, w->ld_y, 0.f, s)
                    : launch_ssd<128, false>(tmBC, tmX, *L, *w, *b, nullptr, 0, y, w->ld_y, 0.f, s);
}

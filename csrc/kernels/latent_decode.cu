// Decode attention on latent pages with tcgen05: one token per sequence, every head of it a row of the same
// MMA, because all heads read the same page rows (latent | rotated key part).
//   S[heads, 64 keys]  = Qabs[heads, width] P[64 keys, width]^T      (SS, K-major, fp32 in TMEM)
//   O[heads, latent]  += softmax weights[heads, 64 keys] P[:, :latent]   (weights from TMEM, pages MN-major)
// The page tile in shared memory serves both products, so a key is read from memory once for all heads.
// One CTA per (range of keys, sequence, 256 latent columns x 128 heads); warp 0 feeds a ring of 64-key tiles,
// page by page through the block table, warp 1 issues the MMAs, warps 2..5 do the softmax of one head per
// thread.  Two score buffers keep the tensor pipe a tile ahead.  Key ranges are merged by a second kernel.
// The query tile holds the rows that are heads and no more: the MMA's further rows read whatever lies behind
// them in shared memory, and their results are never looked at.
#include "../common/host.hpp"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"
#include "../serve/hybrid.hpp"

namespace bb {

constexpr int LD_KEYS = 64, LD_SUB = LD_KEYS * 128, LD_ROWS = 128, LD_COLS = 256, LD_MAX_STAGES = 4;
constexpr int LD_SMEM_MAX = 226 * 1024, LD_BARS = 256;

struct LatDecArgs {
  const int *pos, *tables;     // [rows], [rows][max_blocks]
  int max_blocks, bs, window;
  int hq, q_rows, width, kvrp, nsub, stages, vchunks, splits, tmem_cols;   // q_rows: rows of the query tile
  float scale_log2;
  __nv_bfloat16* out;          // [rows, ldo], head h at h kvrp (one key range)
  int ldo;
  float *part_o, *part_ml;     // [rows][heads][splits][kvrp | 2]
  const __nv_bfloat16* gate;   // raw gate of row r, head h at gate[r ldg + h] (null: none)
  int ldg;
  int* err;
};

__global__ void __launch_bounds__(192, 1)
hy_latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmP,
                        const __grid_constant__ LatDecArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int tile_bytes = a.nsub * LD_SUB, q_sub = a.q_rows * 128;
  uint8_t* sQ = smem;
  uint8_t* sP = smem + a.nsub * q_sub;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + a.stages * tile_bytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;                       // [stages]
  uint64_t* k_empty = k_full + LD_MAX_STAGES;        // [stages]
  uint64_t* s_full = k_empty + LD_MAX_STAGES;        // [2]
  uint64_t* p_ready = s_full + 2;                    // [2], 128 arrivals each
  uint64_t* pv_done = p_ready + 2;                   // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, row = blockIdx.y, vc = blockIdx.z % a.vchunks, h0 = (blockIdx.z / a.vchunks) * 128;
  const int last = a.pos[row], first = a.window > 0 ? max(last - a.window + 1, 0) : 0;
  const int t_first = first / LD_KEYS, n_tiles = last / LD_KEYS + 1 - t_first;
  const int t0 = t_first + (int)((long)n_tiles * split / a.splits), t1 = t_first + (int)((long)n_tiles * (split + 1) / a.splits);
  const int n_units = t1 - t0;
  const int v0 = vc * LD_COLS, nv = min(LD_COLS, (a.kvrp - v0 + 15) & ~15);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < LD_MAX_STAGES; ++i) {
      mbar_init(k_full + i, 1);
      mbar_init(k_empty + i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(s_full + i, 1);
      mbar_init(p_ready + i, 128);
      mbar_init(pv_done + i, 1);
    }
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, a.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, tmem_O = tmem + 128;

  if (warp == 0) {
    if (lane == 0 && n_units > 0) {
      mbar_expect_tx(q_full, a.nsub * q_sub);
      for (int c = 0; c < a.nsub; ++c) tma_load_3d(sQ + c * q_sub, &tmQ, q_full, c * 64, h0, row);
      const int* tab = a.tables + (size_t)row * a.max_blocks;
      for (int u = 0; u < n_units; ++u) {
        const int st = u % a.stages;
        if (!mbar_wait(k_empty + st, ((u / a.stages) & 1) ^ 1)) {
          set_error(a.err, ERR_WAIT_PRODUCER);
          break;
        }
        mbar_expect_tx(k_full + st, tile_bytes);
        for (int i = 0; i < LD_KEYS / a.bs; ++i) {
          const int p = ((t0 + u) * LD_KEYS) / a.bs + i;
          const int blk = p * a.bs <= last && p < a.max_blocks ? max(tab[p], 0) : 0;   // dead pages are masked
          for (int c = 0; c < a.nsub; ++c)
            tma_load_2d(sP + st * tile_bytes + c * LD_SUB + i * a.bs * 128, &tmP, k_full + st, c * 64, blk * a.bs);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_units > 0) {
      const uint32_t idesc_s = umma_idesc(1, 1, 1, 0, 0, 128, LD_KEYS), idesc_o = umma_idesc(1, 1, 1, 0, 1, 128, nv);
      const uint32_t aq = smem_u32(sQ), bp = smem_u32(sP);
      const int ksteps = (a.width + 15) / 16;
      bool ok = mbar_wait(q_full, 0);
      auto issue_s = [&](int u) -> bool {
        const int st = u % a.stages;
        if (!mbar_wait(k_full + st, (u / a.stages) & 1)) return false;
        tc_fence_after();
        for (int t = 0; t < ksteps; ++t)
          umma_f16_ss(tmem + (u & 1) * 64, umma_smem_desc(aq + (t / 4) * q_sub + (t % 4) * 32, 16, 1024),
                      umma_smem_desc(bp + st * tile_bytes + (t / 4) * LD_SUB + (t % 4) * 32, 16, 1024), idesc_s, t != 0);
        umma_commit(s_full + (u & 1));
        return true;
      };
      // scores run two tiles ahead where the ring holds a third tile; with two stages, one, so that finishing a
      // tile never waits for the load into the stage it frees
      const int ahead = a.stages > 2 ? 2 : 1;
      for (int u = 0; u < ahead && u < n_units && ok; ++u) ok = issue_s(u);
      if (!ok) set_error(a.err, ERR_WAIT_MMA_FULL);
      for (int u = 0; u < n_units && ok; ++u) {
        const int st = u % a.stages;
        if (!mbar_wait(p_ready + (u & 1), (u >> 1) & 1)) {
          set_error(a.err, ERR_WAIT_MMA_TMEM);
          ok = false;
          break;
        }
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < LD_KEYS / 16; ++t)
          umma_f16_ts(tmem_O, tmem + (u & 1) * 64 + t * 8,
                      umma_smem_desc(bp + st * tile_bytes + vc * 4 * LD_SUB + t * 2048, LD_SUB, 1024), idesc_o, (u | t) != 0);
        umma_commit(pv_done + (u & 1));
        umma_commit(k_empty + st);
        if (u + ahead < n_units && !issue_s(u + ahead)) {
          set_error(a.err, ERR_WAIT_MMA_FULL);
          ok = false;
        }
      }
    }
  } else {
    const int sw = warp & 3, h = h0 + sw * 32 + lane;
    const uint32_t lane_sel = (uint32_t)(sw * 32) << 16;
    const uint32_t tO = tmem_O + lane_sel;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int u = 0; u < n_units; ++u) {
      const uint32_t tS = tmem + (u & 1) * 64 + lane_sel;
      ok = mbar_wait(s_full + (u & 1), (u >> 1) & 1);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      uint32_t r0[32], r1[32];
      tmem_ld32(tS, r0);
      tmem_ld32(tS + 32, r1);
      tmem_wait_ld();
      const int kv0 = (t0 + u) * LD_KEYS, lim = last - kv0, low = first - kv0;
      const bool need_mask = lim < LD_KEYS - 1 || low > 0;     // the same for every head
      const float sc = a.scale_log2;
      if (need_mask || h >= a.hq) {
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          if (h >= a.hq) r0[i] = r1[i] = 0u;         // not a head
          if (i > lim || i < low) r0[i] = 0xff800000u;
          if (i + 32 > lim || i + 32 < low) r1[i] = 0xff800000u;
        }
      }
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 32; i += 4)
#pragma unroll
        for (int q = 0; q < 4; ++q)
          m4[q] = fmaxf(m4[q], fmaxf(__uint_as_float(r0[i + q]) * sc, __uint_as_float(r1[i + q]) * sc));
      const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      const float m_new = mx > m_ref + 8.f ? mx : m_ref;       // lazy: the reference stays while weights are <= 2^8
      const float alpha = m_new == m_ref ? 1.f : (m_ref == -INFINITY ? 0.f : exp2f(m_ref - m_new));
      if (u > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
        ok = mbar_wait(pv_done + ((u - 1) & 1), ((u - 1) >> 1) & 1);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < nv; c += 16) {
          uint32_t r[16];
          tmem_ld16(tO + c, r);
          tmem_wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
          tmem_st16(tO + c, r);
        }
      }
      l *= alpha;
      m_ref = m_new;
      const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
      uint32_t pk[32];
      float ls = 0.f, ls_b = 0.f;
#pragma unroll
      for (int i = 0; i < 32; i += 2) {
        const float a0 = exp2f(fmaf(__uint_as_float(r0[i]), sc, -m_use)), a1 = exp2f(fmaf(__uint_as_float(r0[i + 1]), sc, -m_use));
        const float b0 = exp2f(fmaf(__uint_as_float(r1[i]), sc, -m_use)), b1 = exp2f(fmaf(__uint_as_float(r1[i + 1]), sc, -m_use));
        if (i & 2) ls_b += (a0 + a1) + (b0 + b1);
        else ls += (a0 + a1) + (b0 + b1);
        pk[i >> 1] = pack_bf16x2_alu(a0, a1);
        pk[16 + (i >> 1)] = pack_bf16x2_alu(b0, b1);
      }
      l += ls + ls_b;
      tmem_st32(tS, pk);
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(p_ready + (u & 1));
    }
    if (ok && n_units > 0) {
      ok = mbar_wait(pv_done + ((n_units - 1) & 1), ((n_units - 1) >> 1) & 1);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (!ok) {
      if (lane == 0) set_error(a.err, ERR_WAIT_SOFTMAX);
    } else {
      tc_fence_after();
      const bool one = a.splits == 1;
      float inv = one && l > 0.f ? 1.f / l : 1.f;
      if (one && a.gate && h < a.hq) inv *= sigmoid_as<__nv_bfloat16>(__bfloat162float(a.gate[(size_t)row * a.ldg + h]));
      const size_t part = ((size_t)row * a.hq + min(h, a.hq - 1)) * a.splits + split;
      if (!one && h < a.hq && vc == 0) {
        a.part_ml[part * 2] = m_ref;
        a.part_ml[part * 2 + 1] = l;
      }
#pragma unroll 1
      for (int c = 0; c < nv; c += 16) {
        uint32_t r[16];
        __syncwarp();
        if (n_units > 0) {
          tmem_ld16(tO + c, r);
          tmem_wait_ld();
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) r[i] = 0u;
        }
        if (h >= a.hq) continue;
#pragma unroll
        for (int q = 0; q < 16; q += 8) {
          if (v0 + c + q >= a.kvrp) break;
          float f[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = __uint_as_float(r[q + j]) * inv;
          if (one) store8(a.out + (size_t)row * a.ldo + h * a.kvrp + v0 + c + q, f);
          else store8(a.part_o + part * a.kvrp + v0 + c + q, f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, a.tmem_cols);
  }
}

__global__ void __launch_bounds__(128)
hy_latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                       int ldo, int rows, int hq, int kvrp, int splits, const __nv_bfloat16* __restrict__ gate, int ldg) {
  const int vecs = kvrp / 8;
  const long t = (long)blockIdx.x * 128 + threadIdx.x;
  const long rh = t / vecs;
  if (rh >= (long)rows * hq) return;
  const int v = (int)(t % vecs) * 8, row = (int)(rh / hq), h = (int)(rh % hq);
  const float* ml = part_ml + rh * splits * 2;
  float m = -INFINITY, l = 0.f, acc[8] = {};
  for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[2 * s]);
  for (int s = 0; s < splits; ++s) {
    if (ml[2 * s] == -INFINITY) continue;
    const float w = exp2f(ml[2 * s] - m);
    float f[8];
    load8(part_o + (rh * splits + s) * kvrp + v, f);
    l = fmaf(w, ml[2 * s + 1], l);
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = fmaf(w, f[j], acc[j]);
  }
  float inv = 1.f / l;
  if (gate) inv *= sigmoid_as<__nv_bfloat16>(__bfloat162float(gate[(size_t)row * ldg + h]));
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j] *= inv;
  store8(out + (size_t)row * ldo + h * kvrp + v, acc);
}

}  // namespace bb

using namespace bb;

// Absorbed attention of the decoded rows (bf16): queries w->qa and outputs w->ol from row qa_row0 on.
// BB_ESIZE where the tiles do not reach (page rows wider than nine 64-column tiles, odd page sizes).
BB_API int bb_hy_latent_decode(const BbHyCfg* c, const BbHyLayer* L, const BbHyWork* w, const BbHyBatch* b, int qa_row0,
                               void* stream) {
  const int rows = b->n - b->n_pre;
  if (rows <= 0) return BB_OK;
  LatDecArgs a{};
  a.width = L->kvrp + L->rotp;
  a.nsub = (a.width + 63) / 64;
  a.bs = c->block_size;
  if (c->dtype || a.nsub > 9 || (a.bs != 16 && a.bs != 32 && a.bs != 64)) return BB_ESIZE;
  a.q_rows = L->hq >= LD_ROWS ? LD_ROWS : (L->hq + 7) & ~7;
  const int q_bytes = a.nsub * a.q_rows * 128, tile = a.nsub * LD_SUB;
  a.stages = (LD_SMEM_MAX - 1024 - LD_BARS - q_bytes) / tile;
  if (a.stages < 1) return BB_ESIZE;
  if (a.stages > LD_MAX_STAGES) a.stages = LD_MAX_STAGES;
  a.pos = b->pos + b->n_pre;
  a.tables = b->tables + (size_t)b->ns_pre * b->max_blocks;
  a.max_blocks = b->max_blocks;
  a.window = L->window;
  a.hq = L->hq;
  a.kvrp = L->kvrp;
  a.vchunks = (L->kvrp + LD_COLS - 1) / LD_COLS;
  a.tmem_cols = L->kvrp > 128 ? 512 : 256;
  a.scale_log2 = L->scale * 1.4426950408889634f;
  a.out = static_cast<__nv_bfloat16*>(w->ol) + (size_t)qa_row0 * w->ld_ol;
  a.ldo = w->ld_ol;
  a.part_o = w->part_o;
  a.part_ml = w->part_ml;
  if (L->gate_kind == 1) a.gate = static_cast<const __nv_bfloat16*>(w->proj) + (size_t)b->n_pre * w->ld_proj + L->off_g;
  a.ldg = w->ld_proj;
  a.err = device_error_word();
  // key ranges: enough CTAs to fill the machine, at most one per tile a query can see
  const int per_range = rows * a.vchunks * ((L->hq + 127) / 128);
  const int tiles = ((L->window > 0 ? L->window : b->max_blocks * a.bs) + LD_KEYS - 2) / LD_KEYS + 1;
  int splits = sm_count() / per_range;
  splits = splits > tiles ? tiles : splits;
  a.splits = splits < 1 ? 1 : (splits > w->splits ? w->splits : splits);
  CUtensorMap tq, tp;
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const __nv_bfloat16* qa = static_cast<const __nv_bfloat16*>(w->qa) + (size_t)qa_row0 * w->ld_qa;
  int rc = make_tmap_3d(&tq, bf, 2, qa, a.width, L->hq, rows, (uint64_t)a.width * 2, (uint64_t)w->ld_qa * 2, 64, a.q_rows);
  if (rc) return rc;
  rc = make_tmap_2d(&tp, bf, 2, L->kc, a.width, (uint64_t)w->pool_blocks * a.bs, (uint64_t)a.width * 2, 64, a.bs);
  if (rc) return rc;
  static PerDeviceOnce once;
  const cudaError_t e = ensure_dyn_smem(once, hy_latent_decode_kernel, LD_SMEM_MAX);
  if (e != cudaSuccess) return (int)e;
  cudaStream_t s = (cudaStream_t)stream;
  // the MMA reads 128 rows of every query sub-tile
  const int q_read = (a.nsub - 1) * a.q_rows * 128 + LD_ROWS * 128, ring = q_bytes + a.stages * tile + LD_BARS;
  const int smem = (ring > q_read ? ring : q_read) + 1024;
  hy_latent_decode_kernel<<<dim3(a.splits, rows, a.vchunks * ((L->hq + 127) / 128)), 192,
                            smem, s>>>(tq, tp, a);
  if (a.splits > 1) {
    const long t = (long)rows * L->hq * (L->kvrp / 8);
    hy_latent_merge_kernel<<<(int)((t + 127) / 128), 128, 0, s>>>(w->part_o, w->part_ml, a.out, w->ld_ol, rows, L->hq,
                                                                  L->kvrp, a.splits, a.gate, a.ldg);
  }
  return (int)cudaGetLastError();
}

// Side-by-side bf16 products on tcgen05: C_g[M, N] = A_g[M, K] B_g[N, K]^T for g < groups, where A_g and C_g
// are column ranges of shared row-major buffers (heads of a projection, blocks of a block-diagonal map).
// One CTA per (128 rows, 128 columns, group): warp 0 feeds a ring of 64-wide K slices by TMA, warp 1 issues
// the MMAs into TMEM, warps 2..5 store through shared memory.  K and N are short (a head, a block), so there is one tile per CTA and
// two or three CTAs share an SM.  Columns of a slice past K are zero-filled by the copy.
#include "../common/host.hpp"
#include "../common/ptx.cuh"

namespace bb {

constexpr int GG_STAGES = 2, GG_BM = 128, GG_BN = 128, GG_TILE = 128 * 128;   // bytes of a 128 x 64 slice
constexpr int GG_SMEM = GG_STAGES * 2 * GG_TILE + 1024 + 128;

__global__ void __launch_bounds__(192, 3)
gemm_groups_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB,
                   const __grid_constant__ CUtensorMap tmC, int N, int K, int* err) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + GG_STAGES * 2 * GG_TILE);
  uint64_t* empty = full + GG_STAGES;
  uint64_t* done = empty + GG_STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * GG_BN, m0 = blockIdx.y * GG_BM, g = blockIdx.z;
  const int nk = (K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int i = 0; i < GG_STAGES; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, 1);
    }
    mbar_init(done, 1);
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, GG_BN);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  if (warp == 0) {
    if (lane == 0) {
      for (int k = 0; k < nk; ++k) {
        const int st = k % GG_STAGES, ph = (k / GG_STAGES) & 1;
        if (!mbar_wait(empty + st, ph ^ 1)) {
          set_error(err, ERR_WAIT_PRODUCER);
          break;
        }
        uint8_t* a = smem + st * 2 * GG_TILE;
        mbar_expect_tx(full + st, 2 * GG_TILE);
        tma_load_3d(a, &tmA, full + st, k * 64, m0, g);
        tma_load_3d(a + GG_TILE, &tmB, full + st, k * 64, n0, g);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc(1, 1, 1, 0, 0, GG_BM, GG_BN);
      for (int k = 0; k < nk; ++k) {
        const int st = k % GG_STAGES, ph = (k / GG_STAGES) & 1;
        if (!mbar_wait(full + st, ph)) {
          set_error(err, ERR_WAIT_MMA_FULL);
          break;
        }
        tc_fence_after();
        const uint32_t a = smem_u32(smem + st * 2 * GG_TILE);
#pragma unroll
        for (int t = 0; t < 4; ++t)
          umma_f16_ss(tmem, umma_smem_desc(a + t * 32, 16, 1024), umma_smem_desc(a + GG_TILE + t * 32, 16, 1024), idesc,
                      (k | t) != 0);
        umma_commit(empty + st);
      }
      umma_commit(done);
    }
  } else {
    const int ew = warp & 3;
    bool ok = mbar_wait(done, 0);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) {
      if (lane == 0) set_error(err, ERR_WAIT_EPILOGUE);
    } else {
      tc_fence_after();
      // every operand tile has been read: the ring holds the output, 64 columns to a swizzled slab
      const int cols = min(GG_BN, N - n0), r = ew * 32 + lane;
#pragma unroll 1
      for (int c = 0; c * 32 < cols; ++c) {
        uint32_t v[32];
        __syncwarp();
        tmem_ld32(tmem + ((uint32_t)(ew * 32) << 16) + c * 32, v);
        tmem_wait_ld();
        uint8_t* p = smem + (c >> 1) * GG_TILE + r * 128;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          uint4 o;
          o.x = pack_bf16x2(__uint_as_float(v[q * 8 + 0]), __uint_as_float(v[q * 8 + 1]));
          o.y = pack_bf16x2(__uint_as_float(v[q * 8 + 2]), __uint_as_float(v[q * 8 + 3]));
          o.z = pack_bf16x2(__uint_as_float(v[q * 8 + 4]), __uint_as_float(v[q * 8 + 5]));
          o.w = pack_bf16x2(__uint_as_float(v[q * 8 + 6]), __uint_as_float(v[q * 8 + 7]));
          *reinterpret_cast<uint4*>(p + (((c & 1) * 4 + q) ^ (r & 7)) * 16) = o;
        }
      }
      fence_proxy_async_smem();
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (ok && ew == 0 && lane == 0) {
      for (int c = 0; c * 64 < N - n0 && c < GG_BN / 64; ++c) tma_store_3d(&tmC, smem + c * GG_TILE, n0 + c * 64, m0, g);
      tma_store_commit();
      tma_store_wait<0>();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, GG_BN);
  }
}

}  // namespace bb

// a_step / c_step: elements between the column ranges of successive groups in A / C; B: [groups][N][K].
// N, K, the steps and the pitches are multiples of 8.
BB_API int bb_gemm_bf16_groups(const void* A, const void* B, void* C, int M, int N, int K, int groups, int lda, int a_step,
                               int ldc, int c_step, void* stream) {
  using namespace bb;
  if (M <= 0 || N <= 0 || K <= 0 || groups <= 0 || groups > 65535) return BB_EARG;
  if (N % 8 || K % 8 || lda % 8 || a_step % 8 || ldc % 8 || c_step % 8) return BB_EARG;
  CUtensorMap ta, tb, tc;
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  int rc = make_tmap_3d(&ta, bf, 2, A, K, M, groups, (uint64_t)lda * 2, (uint64_t)a_step * 2, 64, GG_BM);
  if (rc) return rc;
  rc = make_tmap_3d(&tb, bf, 2, B, K, N, groups, (uint64_t)K * 2, (uint64_t)N * K * 2, 64, GG_BN);
  if (rc) return rc;
  rc = make_tmap_3d(&tc, bf, 2, C, N, M, groups, (uint64_t)ldc * 2, (uint64_t)c_step * 2, 64, GG_BM);
  if (rc) return rc;
  static PerDeviceOnce once;
  const cudaError_t e = ensure_dyn_smem(once, gemm_groups_kernel, GG_SMEM);
  if (e != cudaSuccess) return (int)e;
  gemm_groups_kernel<<<dim3((N + GG_BN - 1) / GG_BN, (M + GG_BM - 1) / GG_BM, groups), 192, GG_SMEM, (cudaStream_t)stream>>>(
      ta, tb, tc, N, K, device_error_word());
  return (int)cudaGetLastError();
}

// fp32 GEMM on the CUDA cores (no tensor-core rounding): C[M,N] = alpha A[M,K] B[N,K]^T, or C += that.
// Serves the 32-bit mode of the engines; 64 x 64 tiles, 16-wide k-steps, 4 x 4 outputs per thread.  Several
// products of equal shape (one per head, one per diagonal block) run side by side along the grid's z.
#include "../common/host.hpp"

namespace bb {

constexpr int SG_T = 64, SG_K = 16;

__global__ void __launch_bounds__(256)
sgemm_kernel(const float* __restrict__ A, const float* __restrict__ B, float* __restrict__ C, int M, int N, int K, int lda,
             int ldb, int ldc, float alpha, int accumulate, size_t a_step, size_t b_step, size_t c_step,
             const int* __restrict__ row_group) {
  A += blockIdx.z * a_step;
  B += blockIdx.z * b_step;
  C += blockIdx.z * c_step;
  if (row_group) {                     // 128 rows share one of several B
    const int g = row_group[blockIdx.y * SG_T / 128];
    if (g < 0) return;
    B += g * b_step;
  }
  __shared__ float sa[SG_K][SG_T + 4], sb[SG_K][SG_T + 4];
  const int m0 = blockIdx.y * SG_T, n0 = blockIdx.x * SG_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // row of the tile, first of four k
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_K) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      sa[lk + j][lr] = (m0 + lr < M && k < K) ? A[(size_t)(m0 + lr) * lda + k] : 0.f;
      sb[lk + j][lr] = (n0 + lr < N && k < K) ? B[(size_t)(n0 + lr) * ldb + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float* c = C + (size_t)m * ldc + n;
      *c = accumulate ? fmaf(alpha, acc[i][j], *c) : alpha * acc[i][j];
    }
  }
}

}  // namespace bb

BB_API int bb_sgemm(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, float alpha,
                    int accumulate, void* stream) {
  using namespace bb;
  if (M <= 0 || N <= 0 || K <= 0) return BB_EARG;
  sgemm_kernel<<<dim3((N + SG_T - 1) / SG_T, (M + SG_T - 1) / SG_T), 256, 0, (cudaStream_t)stream>>>(
      A, B, C, M, N, K, lda, ldb, ldc, alpha, accumulate, 0, 0, 0, nullptr);
  return (int)cudaGetLastError();
}

// C_g = A_g B_g^T for g < groups: A_g starts a_step elements after A_(g-1), C_g c_step after C_(g-1), B holds
// [groups][N][K].
BB_API int bb_sgemm_groups(const float* A, const float* B, float* C, int M, int N, int K, int groups, int lda, int a_step,
                           int ldc, int c_step, void* stream) {
  using namespace bb;
  if (M <= 0 || N <= 0 || K <= 0 || groups <= 0) return BB_EARG;
  sgemm_kernel<<<dim3((N + SG_T - 1) / SG_T, (M + SG_T - 1) / SG_T, groups), 256, 0, (cudaStream_t)stream>>>(
      A, B, C, M, N, K, lda, K, ldc, 1.f, 0, a_step, (size_t)N * K, c_step, nullptr);
  return (int)cudaGetLastError();
}

// C = A B_g^T per 128 rows, g = tile_group[row / 128] (negative: skipped); B: [groups][N][K].
BB_API int bb_sgemm_tiles(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldc, const int* tile_group,
                          void* stream) {
  using namespace bb;
  if (M <= 0 || N <= 0 || K <= 0 || M % 128) return BB_EARG;
  sgemm_kernel<<<dim3((N + SG_T - 1) / SG_T, M / SG_T), 256, 0, (cudaStream_t)stream>>>(A, B, C, M, N, K, lda, K, ldc, 1.f, 0, 0,
                                                                                       (size_t)N * K, 0, tile_group);
  return (int)cudaGetLastError();
}

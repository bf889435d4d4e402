// fp32 values as tensor-core operands of two bf16 terms: the value, and what rounding left over (16 bits of mantissa).
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace bb {

__device__ __forceinline__ float2 split_pair(float a, float b) {
  // packed bf16 pair of the values, packed pair of what rounding left over
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  return make_float2(__uint_as_float(*reinterpret_cast<const uint32_t*>(&h)),
                     __uint_as_float(*reinterpret_cast<const uint32_t*>(&l)));
}

// Byte offset of (row, col) in a swizzled tile whose 64-column sub-tiles lie `sub` bytes apart; col a multiple of 8.
__device__ __forceinline__ int swizzled(int row, int col, int sub) {
  return (col >> 6) * sub + row * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4);
}

// N fp32 values (a multiple of 8) of row `row`, columns col0.. (a multiple of 8), as two terms into two swizzled tiles.
template <int N>
__device__ __forceinline__ void store_split(uint8_t* hi, uint8_t* lo, int row, int col0, const float (&v)[N], int sub) {
#pragma unroll
  for (int q = 0; q < N / 8; ++q) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 t = split_pair(v[q * 8 + 2 * k], v[q * 8 + 2 * k + 1]);
      h[k] = __float_as_uint(t.x);
      l[k] = __float_as_uint(t.y);
    }
    const int o = swizzled(row, col0 + q * 8, sub);
    *reinterpret_cast<uint4*>(hi + o) = make_uint4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<uint4*>(lo + o) = make_uint4(l[0], l[1], l[2], l[3]);
  }
}

}  // namespace bb

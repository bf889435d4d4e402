// Helpers of the row kernels that exist for bf16 and fp32 activations: eight-element loads / stores
// with fp32 arithmetic in between, block sums in a fixed order, and the scalar functions of the
// hybrid layers.
#pragma once
#include <cuda_bf16.h>
#include <math.h>

#include "vec.cuh"

namespace bb {

__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  unpack8(*reinterpret_cast<const bf16x8*>(p), f);
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<bf16x8*>(p) = pack8(f);
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }

// Sum over the block, the same value in every thread; `buf` holds 32 floats.  Two calls in a row
// need different buffers (or a barrier between them).
__device__ __forceinline__ float block_sum(float v, float* buf) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int nw = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) buf[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < nw; ++w) s += buf[w];
  return s;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// The hardware's approximations (2^-22) with tiny arguments flushed: no code around them for denormals.
__device__ __forceinline__ float exp2_hw(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_hw(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rsqrt_hw(float x) {
  float y;
  asm("rsqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float exp_hw(float x) { return exp2_hw(x * kLog2e); }

// Activations whose result is stored as T: with bf16 the exponential and the division are the hardware's
// approximations (far below the rounding that follows), with fp32 they are exact.  An exponential that
// overflows gives a reciprocal of 0, which is the limit of either function there.
template <typename T>
__device__ __forceinline__ float sigmoid_as(float x) {
  if constexpr (sizeof(T) == 2) return rcp_hw(1.f + exp2_hw(-kLog2e * x));
  else return sigmoid_f(x);
}
template <typename T>
__device__ __forceinline__ float silu_as(float x) {
  if constexpr (sizeof(T) == 2) return x * rcp_hw(1.f + exp2_hw(-kLog2e * x));
  else return silu_f(x);
}

// gelu in its tanh form.
template <typename T>
__device__ __forceinline__ float gelu_as(float z) {
  const float t = 0.79788456080286536f * fmaf(0.044715f * z * z, z, z);   // sqrt(2 / pi) (z + 0.044715 z^3)
  if constexpr (sizeof(T) == 2) return z * rcp_hw(1.f + exp2_hw(-2.f * kLog2e * t));
  else return 0.5f * z * (1.f + tanhf(t));
}

// Clamped gated unit: g' = min(g, limit), u' = clamp(u, +-limit); g' sigmoid(alpha g') (u' + shift).
template <typename T>
__device__ __forceinline__ float clamped_glu_as(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_as<T>(alpha * g) * (u + shift);
}

}  // namespace bb

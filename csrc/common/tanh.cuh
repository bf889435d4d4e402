// tanh to fp32 accuracy in translation units compiled with fast math (whose tanhf is the 11-bit
// instruction): the odd Taylor polynomial to u^11 below 0.4 (truncation 6e-8 relative there),
// 1 - 2 / (1 + e^2u) above.
#pragma once
#include <math.h>

namespace bb {

__device__ __forceinline__ float tanh_small(float u) {
  const float s = u * u;
  float p = fmaf(s, -1382.f / 155925.f, 62.f / 2835.f);
  p = fmaf(s, p, -17.f / 315.f);
  p = fmaf(s, p, 2.f / 15.f);
  p = fmaf(s, p, -1.f / 3.f);
  return fmaf(u * s, p, u);
}
__device__ __forceinline__ float tanh_fp32(float u) {
  const float a = fabsf(u);
  if (a < 0.4f) return tanh_small(u);
  return copysignf(1.f - __fdividef(2.f, 1.f + exp2f(fminf(a, 40.f) * 2.885390081777927f)), u);
}

}  // namespace bb

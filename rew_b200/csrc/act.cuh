// Activations shared by the kernels that apply one.
#pragma once
#include <math.h>

namespace rewb {

// z sigmoid(z)
__device__ __forceinline__ float silu_act(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_act(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_act(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// 0.5 z (1 + tanh(w)) = z sigmoid(2 w), w = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_act(float z) { return z / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * z, z * z, z))); }
// The same to a few units in the last place, for results that are stored in 16 bits or meet sums of such
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
// 1 - e^x for x <= 0, e = e^x: near zero, where the difference would lose digits, by the series
__device__ __forceinline__ float one_minus_exp(float x, float e) {
  const float s = -x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.0f);
  return x > -0.25f ? s : 1.0f - e;
}
__device__ __forceinline__ float sqrt_fast(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gelu_tanh_fast(float z) { return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * fmaf(0.044715f * z, z * z, z))); }

}  // namespace rewb

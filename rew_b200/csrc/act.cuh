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
__device__ __forceinline__ float gelu_tanh_fast(float z) { return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * fmaf(0.044715f * z, z * z, z))); }

}  // namespace rewb

// Activation functions shared by the kernels that apply them in an epilogue or on their own (fp32 arithmetic).
#pragma once
#include <cuda_runtime.h>

namespace b200 {

// a_pos z^2 + z / 2 for z > 0, a_neg (exp(z) - 1 - z) + z / 2 for z <= 0
__device__ __forceinline__ float xielu(float z, float a_pos, float a_neg) {
  const float n = fminf(z, 0.f);
  return fmaf(z > 0.f ? a_pos * z : 0.5f, z, z > 0.f ? 0.5f * z : a_neg * (expm1f(n) - n));
}

// The same with the hardware exponential (absolute error of exp below 2^-21 for z <= 0): for results that are rounded to bf16.
__device__ __forceinline__ float xielu_fast(float z, float a_pos, float a_neg) {
  const float e = __expf(fminf(z, 0.f));
  return fmaf(z > 0.f ? a_pos * z : 0.5f, z, z > 0.f ? 0.5f * z : a_neg * (e - 1.0f - z));
}

}  // namespace b200

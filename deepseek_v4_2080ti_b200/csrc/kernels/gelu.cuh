// gelu in its tanh form, z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))), written as z sigmoid(2 u): 1 + tanh(u) would lose
// the small values of a negative z.
#pragma once

namespace b200 {

__device__ __forceinline__ float gelu_tanh(float z) {
  const float u = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z / (1.f + expf(-2.f * u));
}

}  // namespace b200

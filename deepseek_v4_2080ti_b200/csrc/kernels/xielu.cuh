// xIELU activation: z > 0: ap z^2 + z / 2, otherwise an (exp(z) - 1 - z) + z / 2.
#pragma once

namespace b200 {

// Coefficients of the activation a GEMM epilogue applies to its fp32 accumulators (bias: fp32 [N] or null).
struct XieluEpilogue {
  const float* bias;
  float ap, an;
  int on;
};

// exp(v) - 1 - v for v <= 0: Taylor series where the difference would cancel (next term below 1e-7 of the value at
// -1/2), the exponential elsewhere.
__device__ __forceinline__ float expm1_minus(float v) {
  float s = 1.f + v * (1.f / 8.f);
  s = 1.f + v * (1.f / 7.f) * s;
  s = 1.f + v * (1.f / 6.f) * s;
  s = 1.f + v * (1.f / 5.f) * s;
  s = 1.f + v * (1.f / 4.f) * s;
  s = 1.f + v * (1.f / 3.f) * s;
  const float series = 0.5f * v * v * s;
  const float direct = exp2f(v * 1.4426950408889634f) - 1.f - v;
  return v > -0.5f ? series : direct;
}
__device__ __forceinline__ float xielu(float v, float ap, float an) {
  return (v > 0.f ? ap * v * v : an * expm1_minus(v)) + 0.5f * v;
}

// The same for results that are stored as bf16: the exponential branch without the series, whose cancellation leaves an
// absolute error of a few 1e-7 (below half a bf16 step of z / 2 wherever that step is larger, negligible elsewhere), in
// two fused multiply-adds around one exponential.
__device__ __forceinline__ float xielu_bf16(float v, float ap, float an) {
  const float pos = fmaf(ap, v, 0.5f) * v;
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fminf(v, 0.f) * 1.4426950408889634f));
  const float neg = fmaf(an, e, fmaf(0.5f - an, v, -an));
  return v > 0.f ? pos : neg;
}

}  // namespace b200

// Gated feed-forward units on fp32 values:  limit <= 0: silu(g) u.  Otherwise the clamped form with a one-plus second
// factor: g = min(g, limit), u = clamp(u, -limit, limit), y = g sigmoid(slope g) (u + 1).
#pragma once

namespace b200 {

struct GluShape {
  float limit, slope;
};

// FAST: approximate division and exponential (results stored as bf16).
template <bool FAST>
__device__ __forceinline__ float glu(float g, float u, const GluShape& s) {
  float slope = 1.f;
  if (s.limit > 0.f) {
    g = fminf(g, s.limit);
    u = fminf(fmaxf(u, -s.limit), s.limit) + 1.f;
    slope = s.slope;
  }
  const float a = FAST ? __fdividef(g, 1.f + __expf(-slope * g)) : g / (1.f + expf(-slope * g));
  return a * u;
}

}  // namespace b200

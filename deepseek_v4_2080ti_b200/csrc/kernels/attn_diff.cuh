// Shared finish of differential attention: per head, o = a1 - lambda a2 over the two softmax maps, normalised by its root
// mean square over the head's `vdim` values, times (1 - diff), times the head's sigmoid gate.
#pragma once

namespace b200 {

struct DiffFinish {
  float lambda, keep, eps, inv_vdim;     // keep = 1 - diff
};

__device__ __forceinline__ float diff_head_scale(float sum_sq, float gate_logit, const DiffFinish& f) {
  return f.keep / sqrtf(sum_sq * f.inv_vdim + f.eps) / (1.f + expf(-gate_logit));
}

}  // namespace b200

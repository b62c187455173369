// Helpers of the gated linear attention kernels.
#pragma once

#include "kernels.h"

namespace orion {

// Sum of the slabs at p in slab order, eight independent loads in flight.
__device__ __forceinline__ float fold_slabs(const float *p, uint32_t splits, size_t stride) {
  float v = 0.f;
  for (uint32_t s0 = 0; s0 < splits; s0 += 8) {
    float x[8];
#pragma unroll
    for (uint32_t s = 0; s < 8; ++s) x[s] = s0 + s < splits ? p[(size_t)(s0 + s) * stride] : 0.f;
#pragma unroll
    for (uint32_t s = 0; s < 8; ++s) v += x[s];
  }
  return v;
}

// log(1 / (1 + e^-z)), without overflow and with full relative accuracy where it is close to zero.
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

}  // namespace orion

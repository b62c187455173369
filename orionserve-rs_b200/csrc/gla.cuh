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
// The same through the fast exponential and logarithm, whose errors are a few 1e-7 where 1 + e is not close to one; there
// log(1 + e) is three terms of its series.
__device__ __forceinline__ float log_sigmoid_fast(float z) {
  const float e = __expf(-fabsf(z));
  return fminf(z, 0.f) - (e < 0.0078125f ? e * (1.f - e * (0.5f - e * (1.f / 3.f))) : __logf(1.f + e));
}
template <typename T>
__device__ __forceinline__ float log_sigmoid_for(float z) {
  if constexpr (sizeof(T) == 2) return log_sigmoid_fast(z);
  else return log_sigmoid(z);
}

}  // namespace orion

// Shared pieces of the delta rule with one decay per key channel (cd_delta_attn in include/cdeep.h).
#pragma once
#include "../../include/cdeep.h"
#include "elem.cuh"

namespace cdeep {

using DeltaParams = cd_delta_attn;

__device__ __forceinline__ int first_position(const DeltaParams& p) { return p.pos_dev ? *p.pos_dev : p.pos0; }
__device__ __forceinline__ float softplus_precise(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// The same on the hardware's exponential and logarithm; the series keeps small results accurate in
// relative terms (its next term is below 2^-24 there).
__device__ __forceinline__ float softplus_fast(float z) {
  const float e = exp2_approx(-fabsf(z) * 1.4426950408889634f);
  const float small = e * (1.f - e * (0.5f - e * (0.33333333f - e * (0.25f - e * 0.2f))));
  return fmaxf(z, 0.f) + (e < 0.03125f ? small : 0.6931471805599453f * log2_approx(1.f + e));
}
__host__ __device__ __forceinline__ int delta_channels(const DeltaParams& p) { return 2 * p.G * p.dkp + p.H * p.dvp; }

}  // namespace cdeep

// Shared pieces of the delta rule with one decay per key channel (cd_delta_attn in include/cdeep.h).
#pragma once
#include "../../include/cdeep.h"
#include "elem.cuh"

namespace cdeep {

using DeltaParams = cd_delta_attn;

__device__ __forceinline__ int first_position(const DeltaParams& p) { return p.pos_dev ? *p.pos_dev : p.pos0; }
__device__ __forceinline__ float softplus_precise(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__host__ __device__ __forceinline__ int delta_channels(const DeltaParams& p) { return 2 * p.G * p.dkp + p.H * p.dvp; }

}  // namespace cdeep

// Shared pieces of latent attention (cd_latent_attn in include/cdeep.h).
#pragma once
#include "../../include/cdeep.h"
#include "elem.cuh"

namespace cdeep {

using LatentParams = cd_latent_attn;

__device__ __forceinline__ int first_position(const LatentParams& p) { return p.pos_dev ? *p.pos_dev : p.pos0; }

}  // namespace cdeep

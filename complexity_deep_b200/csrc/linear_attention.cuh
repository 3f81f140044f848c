// Shared description of gated linear attention with one decay per key channel.
//
//   log a_t = -softplus(-(A2 u_t + b)) / tau          (u = rank-wide inner projection)
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t / sqrt(dk)
//   y_t = out_scale * (o_t / rms(o_t) * w) * silu(gate_t)   per head
//
// The state [B, H, dkp, dvp] is fp32 and carried from call to call.
#pragma once
#include "../../include/cdeep.h"
#include "elem.cuh"

namespace cdeep {

using LinearAttnParams = cd_linear_attn;

// log of sigmoid(z)^(1 / tau)
__device__ __forceinline__ float log_decay_of(float z, float inv_tau) {
  return -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau;
}

template <typename T>
__device__ __forceinline__ float decay_input(const LinearAttnParams& p, const T* u, int channel) {
  const T* w = static_cast<const T*>(p.a2) + static_cast<long long>(channel) * p.rank;
  float z = to_f32(static_cast<const T*>(p.a2_b)[channel]);
  for (int r = 0; r < p.rank; r += 8) {
    float a[8], b[8];
    load8(u + r, a);
    load8(w + r, b);
#pragma unroll
    for (int e = 0; e < 8; ++e) z = fmaf(a[e], b[e], z);
  }
  return z;
}

}  // namespace cdeep

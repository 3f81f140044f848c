// Element access shared by the kernels that exist for two storage types: bf16 (the serving
// precision, fp32 arithmetic inside) and fp32 (everything in 32 bits).
#pragma once
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace cdeep {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float bf_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
__device__ __forceinline__ uint32_t bf_pack(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

// eight consecutive elements (16-byte aligned) as fp32
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) {
  const uint4 w = *reinterpret_cast<const uint4*>(p);
  f[0] = bf_lo(w.x); f[1] = bf_hi(w.x); f[2] = bf_lo(w.y); f[3] = bf_hi(w.y);
  f[4] = bf_lo(w.z); f[5] = bf_hi(w.z); f[6] = bf_lo(w.w); f[7] = bf_hi(w.w);
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(bf16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(bf_pack(f[0], f[1]), bf_pack(f[2], f[3]), bf_pack(f[4], f[5]),
                                            bf_pack(f[6], f[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

// the same eight elements as loaded, for values in flight
template <typename T> struct Raw8;
template <> struct Raw8<bf16> { uint4 w; };
template <> struct Raw8<float> { float4 a, b; };
__device__ __forceinline__ void raw_load(const bf16* p, Raw8<bf16>& r) { r.w = *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ void raw_load(const float* p, Raw8<float>& r) {
  r.a = *reinterpret_cast<const float4*>(p);
  r.b = *reinterpret_cast<const float4*>(p + 4);
}
__device__ __forceinline__ void raw_unpack(const Raw8<bf16>& r, float (&f)[8]) {
  f[0] = bf_lo(r.w.x); f[1] = bf_hi(r.w.x); f[2] = bf_lo(r.w.y); f[3] = bf_hi(r.w.y);
  f[4] = bf_lo(r.w.z); f[5] = bf_hi(r.w.z); f[6] = bf_lo(r.w.w); f[7] = bf_hi(r.w.w);
}
__device__ __forceinline__ void raw_unpack(const Raw8<float>& r, float (&f)[8]) {
  f[0] = r.a.x; f[1] = r.a.y; f[2] = r.a.z; f[3] = r.a.w;
  f[4] = r.b.x; f[5] = r.b.y; f[6] = r.b.z; f[7] = r.b.w;
}

__device__ __forceinline__ float warp_add(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// programmatic dependent launch: wait for the previous kernel of the stream before touching
// memory, then let the next one be scheduled
__device__ __forceinline__ void pdl_enter() {
  asm volatile("griddepcontrol.wait;" ::: "memory");
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float log2_approx(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// exp and log(1 + x) of attention scores: the hardware approximations for bf16 storage (absolute
// error of a score ~1e-7 of its size), the full-precision functions for fp32 storage
template <typename T> __device__ __forceinline__ float score_exp(float x) {
  return sizeof(T) == 2 ? exp2_approx(x * 1.4426950408889634f) : expf(x);
}
template <typename T> __device__ __forceinline__ float score_log1p(float x) {
  return sizeof(T) == 2 ? 0.6931471805599453f * log2_approx(1.0f + x) : log1pf(x);
}

__device__ __forceinline__ float sigmoid_precise(float z) { return 1.0f / (1.0f + expf(-z)); }
// silu for results that are rounded to bf16 (__fdividef returns 0 once the divisor passes 2^126, as silu does)
__device__ __forceinline__ float silu_fast(float g) {
  return __fdividef(g, 1.0f + exp2_approx(-1.4426950408889634f * g));
}
__device__ __forceinline__ float silu_precise(float g) { return g / (1.0f + expf(-g)); }

}  // namespace cdeep

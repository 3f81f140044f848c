// Gated linear attention with per-channel decay: the decode step (one token per sequence: decay,
// state update, head norm and gate in one kernel, bound by the two passes over the state) and the
// token-by-token form for several tokens, which also serves every call in 32-bit storage.  Prompts
// in bf16 take the chunked tensor-core form of linear_attention_chunk.cu.
#include "linear_attention.cuh"
#include "kernels.h"

namespace cdeep {

namespace {

constexpr int kThreads = 256;

// ---------------------------------------------------------------- decode
template <typename T>
__global__ void __launch_bounds__(kThreads)
gla_step_kernel(const LinearAttnParams p) {
  extern __shared__ float sm[];
  pdl_enter();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int dkp = p.dkp, dvp = p.dvp;
  float* sq = sm;                // [dkp]
  float* sk = sq + dkp;          // [dkp]
  float* sa = sk + dkp;          // [dkp]
  float* sv = sa + dkp;          // [dvp]
  float* so = sv + dvp;          // [kThreads * 4] partial outputs
  __shared__ float s_ss[kThreads / 32];
  const long long row = b;
  const T* u = static_cast<const T*>(p.inner) + row * p.ldp;
  for (int c = tid; c < dkp; c += kThreads) {
    sq[c] = to_f32(static_cast<const T*>(p.q)[row * p.ldp + static_cast<long long>(h) * dkp + c]) * p.q_scale;
    sk[c] = to_f32(static_cast<const T*>(p.k)[row * p.ldp + static_cast<long long>(h) * dkp + c]);
    sa[c] = expf(log_decay_of(decay_input<T>(p, u, h * dkp + c), p.inv_tau));
  }
  for (int c = tid; c < dvp; c += kThreads)
    sv[c] = to_f32(static_cast<const T*>(p.v)[row * p.ldp + static_cast<long long>(h) * dvp + c]);
  __syncthreads();

  // columns in groups of four; the rows of the state are dealt to the row groups
  const int cgs = dvp / 4;                 // dvp <= 1024
  const int rgs = kThreads / cgs;
  const int rg = tid / cgs, col = (tid - rg * cgs) * 4;
  float* S = p.state + (static_cast<long long>(b) * p.H + h) * dkp * dvp;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rg < rgs) {
    const float4 v = *reinterpret_cast<const float4*>(sv + col);
#pragma unroll 4
    for (int r = rg; r < dkp; r += rgs) {
      float4* ptr = reinterpret_cast<float4*>(S + static_cast<long long>(r) * dvp + col);
      float4 s = *ptr;
      const float a = sa[r], k = sk[r], q = sq[r];
      s.x = fmaf(a, s.x, k * v.x);
      s.y = fmaf(a, s.y, k * v.y);
      s.z = fmaf(a, s.z, k * v.z);
      s.w = fmaf(a, s.w, k * v.w);
      *ptr = s;
      o.x = fmaf(q, s.x, o.x);
      o.y = fmaf(q, s.y, o.y);
      o.z = fmaf(q, s.z, o.z);
      o.w = fmaf(q, s.w, o.w);
    }
    *reinterpret_cast<float4*>(so + tid * 4) = o;    // = [rg][dvp]
  }
  __syncthreads();
  // sum over the row groups, head norm, gate
  float ss = 0.f;
  for (int c = tid; c < dvp; c += kThreads) {
    float a = 0.f;
    for (int r = 0; r < rgs; ++r) a += so[r * dvp + c];
    sv[c] = a;
    ss += a * a;
  }
  ss = warp_add(ss);
  if ((tid & 31) == 0) s_ss[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) tot += s_ss[w];
  const float r = 1.0f / sqrtf(tot / static_cast<float>(p.dv) + p.eps);
  const T* gate = static_cast<const T*>(p.gate) + row * p.ldp + static_cast<long long>(h) * dvp;
  T* out = static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * dvp;
  for (int c = tid; c < dvp; c += kThreads) {
    const float g = to_f32(gate[c]);
    out[c] = from_f32<T>(sv[c] * r * to_f32(static_cast<const T*>(p.norm_w)[c]) * silu_precise(g) * p.out_scale);
  }
}

// ---------------------------------------------------------------- several tokens
constexpr int kDecayRows = 32;

// A thread keeps its channel's row of a2 in registers (rank <= 8 R8) and takes kDecayRows tokens.
template <typename T, int R8>
__global__ void __launch_bounds__(kThreads)
gla_decay_kernel(const LinearAttnParams p) {
  extern __shared__ float su[];        // [kDecayRows][8 R8]
  pdl_enter();
  const long long rows = static_cast<long long>(p.B) * p.S, row0 = static_cast<long long>(blockIdx.x) * kDecayRows;
  const int n = static_cast<int>(rows - row0 < kDecayRows ? rows - row0 : kDecayRows);
  const int ch = p.H * p.dkp, c = blockIdx.y * kThreads + threadIdx.x;
  for (int x = threadIdx.x; x < n * 8 * R8; x += kThreads) {
    const int t = x / (8 * R8), r = x - t * 8 * R8;
    su[x] = r < p.rank ? to_f32(static_cast<const T*>(p.inner)[(row0 + t) * p.ldp + r]) : 0.f;
  }
  float w[R8 * 8], bias = 0.f;
#pragma unroll
  for (int x = 0; x < R8; ++x) {
    float f[8] = {};
    if (c < ch && x * 8 < p.rank) load8(static_cast<const T*>(p.a2) + static_cast<long long>(c) * p.rank + x * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) w[x * 8 + e] = f[e];
  }
  if (c < ch) bias = to_f32(static_cast<const T*>(p.a2_b)[c]);
  __syncthreads();
  if (c >= ch) return;
  float* out = p.log_decay + row0 * ch + c;
  for (int t = 0; t < n; ++t) {
    float z = bias;
#pragma unroll
    for (int x = 0; x < R8 * 2; ++x) {
      const float4 u = *reinterpret_cast<const float4*>(su + t * 8 * R8 + x * 4);
      z = fmaf(u.x, w[x * 4], z);
      z = fmaf(u.y, w[x * 4 + 1], z);
      z = fmaf(u.z, w[x * 4 + 2], z);
      z = fmaf(u.w, w[x * 4 + 3], z);
    }
    out[static_cast<long long>(t) * ch] = log_decay_of(z, p.inv_tau);
  }
}

// any rank
template <typename T>
__global__ void __launch_bounds__(kThreads)
gla_decay_wide_kernel(const LinearAttnParams p) {
  pdl_enter();
  const int ch = p.H * p.dkp;
  const long long row = blockIdx.x;
  const T* u = static_cast<const T*>(p.inner) + row * p.ldp;
  for (int c = threadIdx.x; c < ch; c += kThreads)
    p.log_decay[row * ch + c] = log_decay_of(decay_input<T>(p, u, c), p.inv_tau);
}

template <typename T>
cudaError_t launch_decay(const LinearAttnParams& p, cudaStream_t st) {
  const long long rows = static_cast<long long>(p.B) * p.S;
  const dim3 grid(static_cast<unsigned>((rows + kDecayRows - 1) / kDecayRows), (p.H * p.dkp + kThreads - 1) / kThreads);
  auto bytes = [](int r8) { return static_cast<size_t>(kDecayRows) * 8 * r8 * sizeof(float); };
  if (p.rank <= 16) return launch_kernel(gla_decay_kernel<T, 2>, grid, dim3(kThreads), bytes(2), st, p);
  if (p.rank <= 32) return launch_kernel(gla_decay_kernel<T, 4>, grid, dim3(kThreads), bytes(4), st, p);
  if (p.rank <= 64) return launch_kernel(gla_decay_kernel<T, 8>, grid, dim3(kThreads), bytes(8), st, p);
  return launch_kernel(gla_decay_wide_kernel<T>, dim3(static_cast<unsigned>(rows)), dim3(kThreads), 0, st, p);
}

constexpr int kSteps = 16;      // tokens staged in shared memory at a time
constexpr int kCols = 32;       // state columns per block

// M rows of the state per thread (dkp <= 32 M), four columns each
template <typename T, int M>
__global__ void __launch_bounds__(kThreads)
gla_sequence_kernel(const LinearAttnParams p) {
  extern __shared__ float sm[];
  pdl_enter();
  const int h = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * kCols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dkp = p.dkp, dvp = p.dvp, ch = p.H * dkp;
  float* sq = sm;                            // [kSteps][dkp]
  float* sk = sq + kSteps * dkp;
  float* sa = sk + kSteps * dkp;
  float* sv = sa + kSteps * dkp;             // [kSteps][kCols]
  float* so = sv + kSteps * kCols;           // [kSteps][8 warps][kCols]
  const int cl = (lane & 7) * 4;             // this thread's columns within the block
  const int rg = warp * 4 + (lane >> 3);     // rows rg, rg + 32, ...
  const bool col_ok = col0 + cl < dvp;       // dvp is a multiple of 8
  float* S = p.state + (static_cast<long long>(b) * p.H + h) * dkp * dvp;
  float4 s[M];
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int r = rg + 32 * m;
    s[m] = (r < dkp && col_ok) ? *reinterpret_cast<const float4*>(S + static_cast<long long>(r) * dvp + col0 + cl)
                               : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const long long row0 = static_cast<long long>(b) * p.S;
  for (int t0 = 0; t0 < p.S; t0 += kSteps) {
    const int n = min(kSteps, p.S - t0);
    for (int idx = tid; idx < n * dkp; idx += kThreads) {
      const int t = idx / dkp, c = idx - t * dkp;
      const long long off = (row0 + t0 + t) * p.ldp + static_cast<long long>(h) * dkp + c;
      sq[idx] = to_f32(static_cast<const T*>(p.q)[off]) * p.q_scale;
      sk[idx] = to_f32(static_cast<const T*>(p.k)[off]);
      sa[idx] = expf(p.log_decay[(row0 + t0 + t) * ch + h * dkp + c]);
    }
    for (int idx = tid; idx < n * kCols; idx += kThreads) {
      const int t = idx / kCols, c = idx - t * kCols;
      sv[idx] = col0 + c < dvp
                    ? to_f32(static_cast<const T*>(p.v)[(row0 + t0 + t) * p.ldp + static_cast<long long>(h) * dvp + col0 + c])
                    : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float4 v = *reinterpret_cast<const float4*>(sv + t * kCols + cl);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int r = rg + 32 * m;
        if (r < dkp) {
          const float a = sa[t * dkp + r], k = sk[t * dkp + r], q = sq[t * dkp + r];
          s[m].x = fmaf(a, s[m].x, k * v.x);
          s[m].y = fmaf(a, s[m].y, k * v.y);
          s[m].z = fmaf(a, s[m].z, k * v.z);
          s[m].w = fmaf(a, s[m].w, k * v.w);
          o.x = fmaf(q, s[m].x, o.x);
          o.y = fmaf(q, s[m].y, o.y);
          o.z = fmaf(q, s[m].z, o.z);
          o.w = fmaf(q, s[m].w, o.w);
        }
      }
#pragma unroll
      for (int d = 8; d < 32; d <<= 1) {
        o.x += __shfl_xor_sync(0xffffffffu, o.x, d);
        o.y += __shfl_xor_sync(0xffffffffu, o.y, d);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, d);
        o.w += __shfl_xor_sync(0xffffffffu, o.w, d);
      }
      if (lane < 8) *reinterpret_cast<float4*>(so + (t * 8 + warp) * kCols + cl) = o;
    }
    __syncthreads();
    for (int idx = tid; idx < n * kCols; idx += kThreads) {
      const int t = idx / kCols, c = idx - t * kCols;
      if (col0 + c < dvp) {
        float a = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) a += so[(t * 8 + w) * kCols + c];
        p.o_raw[(row0 + t0 + t) * (p.H * dvp) + static_cast<long long>(h) * dvp + col0 + c] = a;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int r = rg + 32 * m;
    if (r < dkp && col_ok) *reinterpret_cast<float4*>(S + static_cast<long long>(r) * dvp + col0 + cl) = s[m];
  }
}

// head norm and gate on the raw outputs; one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(kThreads)
gla_finish_kernel(const LinearAttnParams p) {
  pdl_enter();
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(p.B) * p.S * p.H) return;
  const int lane = threadIdx.x & 31;
  const long long row = item / p.H;
  const int h = static_cast<int>(item - row * p.H);
  const float* o = p.o_raw + item * p.dvp;
  const T* gate = static_cast<const T*>(p.gate) + row * p.ldp + static_cast<long long>(h) * p.dvp;
  T* out = static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.dvp;
  float ss = 0.f;
  for (int c = lane; c < p.dvp; c += 32) ss += o[c] * o[c];
  const float r = 1.0f / sqrtf(warp_add(ss) / static_cast<float>(p.dv) + p.eps);
  for (int c = lane; c < p.dvp; c += 32)
    out[c] = from_f32<T>(o[c] * r * to_f32(static_cast<const T*>(p.norm_w)[c]) * silu_precise(to_f32(gate[c])) *
                         p.out_scale);
}

template <typename T>
cudaError_t launch_sequence(const LinearAttnParams& p, cudaStream_t st) {
  const dim3 grid((p.dvp + kCols - 1) / kCols, p.H, p.B), block(kThreads);
  const size_t bytes = (3 * kSteps * p.dkp + kSteps * kCols + kSteps * 8 * kCols) * sizeof(float);
#define CDEEP_GLA_SEQ(M)                                                                                     \
  {                                                                                                          \
    cudaError_t e = cudaFuncSetAttribute(gla_sequence_kernel<T, M>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                         static_cast<int>(bytes));                                           \
    if (e != cudaSuccess) return e;                                                                          \
    return launch_kernel(gla_sequence_kernel<T, M>, grid, block, bytes, st, p);                              \
  }
  if (p.dkp <= 32) CDEEP_GLA_SEQ(1)
  if (p.dkp <= 64) CDEEP_GLA_SEQ(2)
  if (p.dkp <= 128) CDEEP_GLA_SEQ(4)
  if (p.dkp <= 256) CDEEP_GLA_SEQ(8)
  if (p.dkp <= 512) CDEEP_GLA_SEQ(16)
#undef CDEEP_GLA_SEQ
  return cudaErrorInvalidValue;
}

template <typename T>
cudaError_t launch_step(const LinearAttnParams& p, cudaStream_t st) {
  const size_t bytes = (3 * p.dkp + p.dvp + kThreads * 4) * sizeof(float);
  return launch_kernel(gla_step_kernel<T>, dim3(p.H, p.B), dim3(kThreads), bytes, st, p);
}

}  // namespace

bool linear_attention_supported(int dkp, int dvp) { return dkp <= 512 && dvp <= 1024; }

cudaError_t launch_gla_step(const LinearAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0) return cudaSuccess;
  return fp32 ? launch_step<float>(p, st) : launch_step<bf16>(p, st);
}

cudaError_t launch_gla_decay(const LinearAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_decay<float>(p, st) : launch_decay<bf16>(p, st);
}

cudaError_t launch_gla_sequence(const LinearAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_sequence<float>(p, st) : launch_sequence<bf16>(p, st);
}

cudaError_t launch_gla_finish(const LinearAttnParams& p, int fp32, cudaStream_t st) {
  const long long items = static_cast<long long>(p.B) * p.S * p.H;
  if (items == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>((items + 7) / 8));
  return fp32 ? launch_kernel(gla_finish_kernel<float>, grid, dim3(kThreads), 0, st, p)
              : launch_kernel(gla_finish_kernel<bf16>, grid, dim3(kThreads), 0, st, p);
}

}  // namespace cdeep

// Latent attention: the step before it (latent norm, rotation, cache append) and the form that takes
// any sizes and either storage type, one block per query and head.
#include "latent_attention.cuh"
#include "kernels.h"

namespace cdeep {

namespace {

constexpr int kThreads = 128;

// Four interleaved pairs of eight consecutive elements turned by the angles of one position.
__device__ __forceinline__ void turn8(float (&f)[8], const float* cs, const float* sn) {
  const float4 c = *reinterpret_cast<const float4*>(cs), s = *reinterpret_cast<const float4*>(sn);
  const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float u = f[2 * i], v = f[2 * i + 1];
    f[2 * i] = u * cv[i] - v * sv[i];
    f[2 * i + 1] = v * cv[i] + u * sv[i];
  }
}

// One block per projection row: warp 0 norms the latent, the others rotate.
template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_prepare_kernel(const LatentParams p) {
  pdl_enter();
  const int row = blockIdx.x, b = row / p.S, t = row - b * p.S;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = first_position(p) + t;
  if (pos >= p.capacity || pos >= p.positions) return;      // a device-side position past the cache
  T* kv = static_cast<T*>(p.kv) + row * p.ldp;
  T* dst = static_cast<T*>(p.cache) + (static_cast<long long>(b) * p.capacity + pos) * (p.rankp + p.rotp);
  if (warp == 0) {
    float ss = 0.f;
    for (int c = lane * 8; c < p.rankp; c += 256) {
      float f[8];
      load8(kv + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
    }
    const float r = 1.0f / sqrtf(warp_add(ss) / static_cast<float>(p.rank) + p.eps);
    for (int c = lane * 8; c < p.rankp; c += 256) {
      float f[8], w[8];
      load8(kv + c, f);
      load8(static_cast<const T*>(p.norm_w) + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = f[e] * r * w[e];
      store8(kv + c, f);
      store8(dst + c, f);
    }
    return;
  }
  const float* cs = p.cos_t + static_cast<long long>(pos) * (p.rotp / 2);
  const float* sn = p.sin_t + static_cast<long long>(pos) * (p.rotp / 2);
  const int per = p.rotp / 8;
  T* q = static_cast<T*>(p.q) + row * p.ldp;
  for (int i = threadIdx.x - 32; i < (p.H + 1) * per; i += kThreads - 32) {
    const int h = i / per, c = (i - h * per) * 8;
    const bool key = h == p.H;
    T* src = key ? kv + p.rankp + c : q + static_cast<long long>(h) * (p.dimp + p.rotp) + p.dimp + c;
    float f[8];
    load8(src, f);
    turn8(f, cs + c / 2, sn + c / 2);
    store8(key ? dst + p.rankp + c : src, f);
  }
}

constexpr int kKeys = 32;      // keys per step
constexpr int kMaxCols = 8;    // latent elements per thread: rankp <= kThreads * kMaxCols

// One block per (query, head): the query goes to the latent's space, attends to the cached rows, and
// the weighted latent comes back through uv.
template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_rows_kernel(const LatentParams p) {
  extern __shared__ float sm[];
  pdl_enter();
  const int h = blockIdx.y, row = blockIdx.x, b = row / p.S, t = row - b * p.S;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int W = p.rankp + p.rotp;
  float* sq = sm;               // [W]
  float* sd = sq + W;           // [dimp]
  float* ss = sd + p.dimp;      // [kKeys] scores
  float* se = ss + kKeys;       // [kKeys] their exponentials
  const T* q = static_cast<const T*>(p.q) + row * p.ldp + static_cast<long long>(h) * (p.dimp + p.rotp);
  for (int c = tid; c < p.dimp; c += kThreads) sd[c] = to_f32(q[c]);
  for (int c = tid; c < p.rotp; c += kThreads) sq[p.rankp + c] = to_f32(q[p.dimp + c]);
  __syncthreads();
  const T* uk = static_cast<const T*>(p.uk) + static_cast<long long>(h) * p.dimp * p.rankp;
  for (int c = tid; c < p.rankp; c += kThreads) {
    float a = 0.f;
    for (int d = 0; d < p.dim; ++d) a = fmaf(sd[d], to_f32(uk[static_cast<long long>(d) * p.rankp + c]), a);
    sq[c] = a;
  }
  __syncthreads();
  const int len = min(first_position(p) + t + 1, p.capacity);
  const T* cache = static_cast<const T*>(p.cache) + static_cast<long long>(b) * p.capacity * W;
  float m = -INFINITY, l = 0.f, acc[kMaxCols] = {};
  for (int j0 = 0; j0 < len; j0 += kKeys) {
    for (int x = warp; x < kKeys; x += kThreads / 32) {
      float s = 0.f;
      if (j0 + x < len) {
        const T* key = cache + static_cast<long long>(j0 + x) * W;
        for (int c = lane * 8; c < W; c += 256) {
          float f[8];
          load8(key + c, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) s = fmaf(f[e], sq[c + e], s);
        }
      }
      s = warp_add(s);
      if (lane == 0) ss[x] = j0 + x < len ? s * p.scale : -INFINITY;
    }
    __syncthreads();
    const float m_new = fmaxf(m, warp_max(ss[lane]));
    const float f = expf(m - m_new);
    const float e = expf(ss[lane] - m_new);
    l = l * f + warp_add(e);
    m = m_new;
    if (warp == 0) se[lane] = e;
    __syncthreads();
    const int n = min(kKeys, len - j0);
#pragma unroll
    for (int x = 0; x < kMaxCols; ++x) {
      const int c = tid + x * kThreads;
      acc[x] *= f;
      if (c < p.rankp)
        for (int k = 0; k < n; ++k)
          acc[x] = fmaf(se[k], to_f32(cache[static_cast<long long>(j0 + k) * W + c]), acc[x]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int x = 0; x < kMaxCols; ++x) {
    const int c = tid + x * kThreads;
    if (c < p.rankp) sq[c] = acc[x] / l;
  }
  __syncthreads();
  const float g = sigmoid_precise(to_f32(static_cast<const T*>(p.gate)[row * p.ldp + h])) * p.out_scale;
  T* out = static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.vp;
  const T* uv = static_cast<const T*>(p.uv) + static_cast<long long>(h) * p.vp * p.rankp;
  for (int v = warp; v < p.vp; v += kThreads / 32) {
    float a = 0.f;
    for (int c = lane * 8; c < p.rankp; c += 256) {
      float f[8];
      load8(uv + static_cast<long long>(v) * p.rankp + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) a = fmaf(f[e], sq[c + e], a);
    }
    a = warp_add(a);
    if (lane == 0) out[v] = from_f32<T>(a * g);
  }
}

template <typename T>
cudaError_t launch_rows(const LatentParams& p, cudaStream_t st) {
  const size_t bytes = (p.rankp + p.rotp + p.dimp + 2 * kKeys) * sizeof(float);
  return launch_kernel(latent_rows_kernel<T>, dim3(p.B * p.S, p.H), dim3(kThreads), bytes, st, p);
}

}  // namespace

bool latent_rows_supported(const LatentParams& p) {
  return p.rankp <= kThreads * kMaxCols && p.dimp <= 1024 && p.rotp <= 1024 && p.H <= 65535;
}

cudaError_t launch_latent_prepare(const LatentParams& p, int fp32, cudaStream_t st) {
  const long long rows = static_cast<long long>(p.B) * p.S;
  if (rows == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>(rows)), block(kThreads);
  return fp32 ? launch_kernel(latent_prepare_kernel<float>, grid, block, 0, st, p)
              : launch_kernel(latent_prepare_kernel<bf16>, grid, block, 0, st, p);
}

cudaError_t launch_latent_rows(const LatentParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_rows<float>(p, st) : launch_rows<bf16>(p, st);
}

}  // namespace cdeep

// Learned routing: the choice of experts per token, the gather of the chosen rows into expert order,
// and the weighted sum of the experts' results into the fp32 stream.
#include "elem.cuh"
#include "kernels.h"

namespace cdeep {

namespace {

constexpr int kThreads = 256;
constexpr int kMaxExperts = 128;
constexpr int kPer = kMaxExperts / 32;

// the largest of v over the warp and its index; the lower index wins a tie
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}

// one warp per token; lane l holds experts l, l + 32, ...
__global__ void __launch_bounds__(kThreads)
route_top_kernel(const float* __restrict__ logits, long long ld, int T, int E, int count, int keep, int top,
                 long long* __restrict__ ids, float* __restrict__ weights) {
  __shared__ float s_all[kThreads / 32][kMaxExperts];
  __shared__ unsigned char s_ok[kThreads / 32][kMaxExperts];
  pdl_enter();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * (kThreads / 32) + warp;
  if (t >= T) return;
  float s[kPer], m = -INFINITY, sum = 0.f;
#pragma unroll
  for (int x = 0; x < kPer; ++x) {
    const int e = lane + 32 * x;
    s[x] = e < E ? logits[t * ld + e] : -INFINITY;
    m = fmaxf(m, s[x]);
  }
  m = warp_max(m);
#pragma unroll
  for (int x = 0; x < kPer; ++x) sum += lane + 32 * x < E ? expf(s[x] - m) : 0.f;
  sum = warp_add(sum);
  const int size = E / count;
  if (keep < count) {
#pragma unroll
    for (int x = 0; x < kPer; ++x)
      if (lane + 32 * x < E) s_all[warp][lane + 32 * x] = s[x];
    __syncwarp();
    float gv[kPer];                          // best logit of groups lane, lane + 32, ...
#pragma unroll
    for (int x = 0; x < kPer; ++x) {
      const int g = lane + 32 * x;
      gv[x] = -INFINITY;
      if (g < count) {
        s_ok[warp][g] = 0;
        for (int e = g * size; e < (g + 1) * size; ++e) gv[x] = fmaxf(gv[x], s_all[warp][e]);
      }
    }
    __syncwarp();
    unsigned taken = 0;
    for (int k = 0; k < keep; ++k) {
      float v = -INFINITY;
      int i = kMaxExperts;
#pragma unroll
      for (int x = 0; x < kPer; ++x) {
        const int g = lane + 32 * x;
        if (g < count && !((taken >> x) & 1u) && (i == kMaxExperts || gv[x] > v)) {
          v = gv[x];
          i = g;
        }
      }
      warp_best(v, i);
      if (i < kMaxExperts && (i & 31) == lane) {
        taken |= 1u << (i >> 5);
        s_ok[warp][i] = 1;
      }
    }
    __syncwarp();
#pragma unroll
    for (int x = 0; x < kPer; ++x) {
      const int e = lane + 32 * x;
      if (e < E && !s_ok[warp][e / size]) s[x] = -INFINITY;
    }
  }
  unsigned taken = 0;
  float chosen = 0.f, mine = 0.f;            // lane k keeps the weight of choice k (top <= 128: lane + 32 x)
  float keep_w[kPer] = {};
  int keep_i[kPer] = {};
  for (int k = 0; k < top; ++k) {
    float v = -INFINITY;
    int i = kMaxExperts;
#pragma unroll
    for (int x = 0; x < kPer; ++x) {
      const int e = lane + 32 * x;
      if (e < E && !((taken >> x) & 1u) && s[x] > -INFINITY && (i == kMaxExperts || s[x] > v)) {
        v = s[x];
        i = e;
      }
    }
    warp_best(v, i);
    i = min(i, E - 1);                       // logits that are not numbers leave nothing to choose
    if ((i & 31) == lane) taken |= 1u << (i >> 5);
    mine = expf(v - m) / sum;
    chosen += mine;
#pragma unroll
    for (int x = 0; x < kPer; ++x)
      if (k == lane + 32 * x) {
        keep_w[x] = mine;
        keep_i[x] = i;
      }
  }
#pragma unroll
  for (int x = 0; x < kPer; ++x) {
    const int k = lane + 32 * x;
    if (k < top) {
      ids[static_cast<long long>(t) * top + k] = keep_i[x];
      weights[static_cast<long long>(t) * top + k] = keep_w[x] / (chosen + 1e-20f);
    }
  }
}

// one warp per row
__global__ void __launch_bounds__(kThreads)
gather_div_kernel(const uint4* __restrict__ x, const int* __restrict__ perm, int div, uint4* __restrict__ out,
                  long long n, int rows, int vecs) {
  pdl_enter();
  const long long i = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (i >= n) return;
  const int src = min(max(perm[i] / div, 0), rows - 1);
  const uint4* s = x + static_cast<long long>(src) * vecs;
  uint4* d = out + i * vecs;
  for (int c = threadIdx.x & 31; c < vecs; c += 32) d[c] = s[c];
}

// one block per token
template <typename T>
__global__ void __launch_bounds__(128)
combine_top_kernel(const T* __restrict__ y, const int* __restrict__ inv_perm, const float* __restrict__ weights, int top,
                   float scale, float* __restrict__ x, int rows, int ldx) {
  pdl_enter();
  const long long t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < ldx; c += 128 * 8) {
    float acc[8] = {};
    for (int j = 0; j < top; ++j) {
      const int r = min(max(inv_perm[t * top + j], 0), rows - 1);
      const float w = weights[t * top + j];
      float f[8];
      load8(y + static_cast<long long>(r) * ldx + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(w, f[e], acc[e]);
    }
    float f[8];
    load8(x + t * ldx + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = fmaf(scale, acc[e], f[e]);
    store8(x + t * ldx + c, f);
  }
}

}  // namespace

cudaError_t launch_route_top(const float* logits, long long ld, int T, int E, int count, int keep, int top,
                             long long* ids, float* weights, cudaStream_t st) {
  if (T == 0) return cudaSuccess;
  return launch_kernel(route_top_kernel, dim3((T + 7) / 8), dim3(kThreads), 0, st, logits, ld, T, E, count, keep, top, ids,
                       weights);
}

cudaError_t launch_gather_div(const void* x, const int* perm, int div, void* out, long long n, int rows, int row_bytes,
                              cudaStream_t st) {
  if (n == 0) return cudaSuccess;
  return launch_kernel(gather_div_kernel, dim3(static_cast<unsigned>((n + 7) / 8)), dim3(kThreads), 0, st,
                       static_cast<const uint4*>(x), perm, div, static_cast<uint4*>(out), n, rows, row_bytes / 16);
}

cudaError_t launch_combine_top(const void* y, const int* inv_perm, const float* weights, int top, float scale, float* x,
                               int T, int ldx, int fp32, cudaStream_t st) {
  if (T == 0) return cudaSuccess;
  return fp32 ? launch_kernel(combine_top_kernel<float>, dim3(T), dim3(128), 0, st, static_cast<const float*>(y), inv_perm,
                              weights, top, scale, x, T * top, ldx)
              : launch_kernel(combine_top_kernel<bf16>, dim3(T), dim3(128), 0, st, static_cast<const bf16*>(y), inv_perm,
                              weights, top, scale, x, T * top, ldx);
}

}  // namespace cdeep

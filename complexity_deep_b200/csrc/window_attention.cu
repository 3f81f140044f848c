// Sliding-window attention with kept first tokens, distance bias and head mixing: the per-head
// norm, the ring append, and the kernel that handles one query per thread-block cluster.  The
// latter serves prompts in 32-bit storage and head layouts that the kernels of
// window_attention_prefill.cu (prompts in bf16) and window_attention_decode.cu do not take.
#include <cfloat>
#include <cooperative_groups.h>
#include "kernels.h"
#include "window_attention.cuh"

namespace cg = cooperative_groups;

namespace cdeep {

namespace {

constexpr int kThreads = 256;
constexpr int kRep = 4;          // query heads of a group handled together

// q and k heads of every row in place: x / rms(x) * w, mean over `dim` columns.  LPH lanes per head,
// eight columns per lane and round.
template <typename T, int LPH>
__global__ void __launch_bounds__(256)
head_norm_kernel(const WindowAttnParams p) {
  pdl_enter();
  const int heads = p.H + p.G;
  const long long item = (blockIdx.x * 256ll + threadIdx.x) / LPH;
  const bool ok = item < static_cast<long long>(p.B) * p.S * heads;
  const int sub = threadIdx.x % LPH;
  const long long row = ok ? item / heads : 0;
  const int h = ok ? static_cast<int>(item - row * heads) : 0;
  const bool is_q = h < p.H;
  T* x = static_cast<T*>(is_q ? p.q : p.k) + row * p.ldp + static_cast<long long>(is_q ? h : h - p.H) * p.dp;
  const T* w = static_cast<const T*>(is_q ? p.q_w : p.k_w);
  float ss = 0.f;
  for (int c = sub * 8; c < p.dp; c += LPH * 8) {
    float f[8];
    load8(x + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
  }
#pragma unroll
  for (int d = 1; d < LPH; d <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
  if (!ok) return;
  for (int c = sub * 8; c < p.dp; c += LPH * 8) {
    float f[8], wv[8];
    load8(x + c, f);
    load8(w + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= r * wv[e];
    store8(x + c, f);
  }
}

template <typename T>
cudaError_t head_norm_any(const WindowAttnParams& p, cudaStream_t st) {
  const long long items = static_cast<long long>(p.B) * p.S * (p.H + p.G);
  auto grid = [&](int lph) { return dim3(static_cast<unsigned>((items * lph + 255) / 256)); };
  if (p.dp <= 64) return launch_kernel(head_norm_kernel<T, 8>, grid(8), dim3(256), 0, st, p);
  if (p.dp <= 128) return launch_kernel(head_norm_kernel<T, 16>, grid(16), dim3(256), 0, st, p);
  return launch_kernel(head_norm_kernel<T, 32>, grid(32), dim3(256), 0, st, p);
}

// Rows of the call that later queries may see go into the ring: the kept first positions and the
// last `window` ones.  One block per (row, sequence).
template <typename T>
__global__ void __launch_bounds__(128)
window_append_kernel(const WindowAttnParams p) {
  pdl_enter();
  const int t = blockIdx.x, b = blockIdx.y;
  const int pos0 = window_pos0(p);
  const int j = pos0 + t;
  if (j >= p.keep && j + p.window < pos0 + p.S) return;   // overwritten by a later row of this call
  const long long slot = static_cast<long long>(b) * (p.keep + p.window) + window_slot(j, p.window, p.keep);
  const long long row = static_cast<long long>(b) * p.S + t;
  const int nk = p.G * p.dp, nv = p.G * p.vp;
  const T* k = static_cast<const T*>(p.k) + row * p.ldp;
  const T* v = static_cast<const T*>(p.v) + row * p.ldp;
  T* rk = static_cast<T*>(p.ring_k) + slot * nk;
  T* rv = static_cast<T*>(p.ring_v) + slot * nv;
  for (int c = threadIdx.x * 8; c < nk + nv; c += blockDim.x * 8) {
    float f[8];
    if (c < nk) {
      load8(k + c, f);
      store8(rk + c, f);
    } else {
      load8(v + c - nk, f);
      store8(rv + c - nk, f);
    }
  }
}

struct RowsSmem {   // offsets in floats
  int q, s, m, stat, o, red, total;
};
__host__ __device__ inline RowsSmem rows_smem(int H, int dp, int vp, int cap) {
  RowsSmem L;
  L.q = 0;                                  // [H][dp]
  L.s = L.q + H * dp;                       // [H][cap] scores, then weights
  L.m = L.s + H * cap;                      // [H][cap] mixed weights
  L.stat = L.m + H * cap;                   // [2][H] this block's maximum and sum
  L.o = L.stat + ((2 * H + 3) & ~3);        // [H][vp] this block's part of the output
  L.red = L.o + H * vp;                     // [kThreads][kRep * 8]
  L.total = L.red + kThreads * kRep * 8;
  return L;
}

// One query per cluster of `gridDim.x / S` blocks; the blocks share the query's keys and exchange
// their softmax statistics and parts of the output through distributed shared memory.
template <typename T>
__global__ void __launch_bounds__(kThreads)
window_rows_kernel(const WindowAttnParams p, int cap) {
  extern __shared__ float4 smem4[];
  float* sm = reinterpret_cast<float*>(smem4);
  pdl_enter();
  cg::cluster_group cluster = cg::this_cluster();
  const int CL = static_cast<int>(cluster.num_blocks());
  const int rank = static_cast<int>(cluster.block_rank());
  const int t = blockIdx.x / CL, b = blockIdx.y;
  const int H = p.H, G = p.G, rep = H / G, dp = p.dp, vp = p.vp;
  const RowsSmem L = rows_smem(H, dp, vp, cap);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos0 = window_pos0(p);
  const int i = pos0 + t;
  const long long row = static_cast<long long>(b) * p.S + t;
  const WindowKeys keys(i, p.window, p.keep);
  const int count = keys.kept + (i - keys.first + 1);
  const int chunk = (count + CL - 1) / CL;
  const int n0 = min(rank * chunk, count);
  const int nk = min(chunk, count - n0);        // keys of this block (0 possible)

  // queries, pre-scaled
  const T* qrow = static_cast<const T*>(p.q) + row * p.ldp;
  for (int c = tid; c < H * dp; c += kThreads) sm[L.q + c] = to_f32(qrow[c]) * p.scale;
  __syncthreads();

  const long long slots = p.keep + p.window;
  const T* ring_k = static_cast<const T*>(p.ring_k) + b * slots * G * dp;
  const T* ring_v = static_cast<const T*>(p.ring_v) + b * slots * G * vp;
  const T* new_k = static_cast<const T*>(p.k) + static_cast<long long>(b) * p.S * p.ldp;
  const T* new_v = static_cast<const T*>(p.v) + static_cast<long long>(b) * p.S * p.ldp;

  // scores: a thread takes one (key, key head) pair and all query heads of the group
  for (int item = tid; item < nk * G; item += kThreads) {
    const int c = item / nk, n = item - c * nk;
    const int j = keys.position(n0 + n);
    const T* kp = j >= pos0 ? new_k + (j - pos0) * p.ldp + static_cast<long long>(c) * dp
                            : ring_k + (static_cast<long long>(window_slot(j, p.window, p.keep)) * G + c) * dp;
    const float dist = static_cast<float>(i - j);
    for (int r0 = 0; r0 < rep; r0 += kRep) {
      float acc[kRep] = {};
      for (int d = 0; d < dp; d += 8) {
        float f[8];
        load8(kp + d, f);
#pragma unroll
        for (int r = 0; r < kRep; ++r) {
          if (r0 + r < rep) {
            const float4* qv = reinterpret_cast<const float4*>(sm + L.q + (c * rep + r0 + r) * dp + d);
            const float4 a = qv[0], bq = qv[1];
            acc[r] += f[0] * a.x + f[1] * a.y + f[2] * a.z + f[3] * a.w + f[4] * bq.x + f[5] * bq.y + f[6] * bq.z +
                      f[7] * bq.w;
          }
        }
      }
#pragma unroll
      for (int r = 0; r < kRep; ++r) {
        if (r0 + r < rep) {
          const int h = c * rep + r0 + r;
          const float r1 = to_f32(static_cast<const T*>(p.r1)[h]), r2 = to_f32(static_cast<const T*>(p.r2)[h]);
          sm[L.s + h * cap + n] = acc[r] - r1 * log1pf(r2 * dist);
        }
      }
    }
  }
  __syncthreads();

  // softmax statistics of this block's keys, then of the whole cluster
  for (int h = warp; h < H; h += kThreads / 32) {
    float m = -FLT_MAX, l = 0.f;
    for (int n = lane; n < nk; n += 32) m = fmaxf(m, sm[L.s + h * cap + n]);
    m = warp_max(m);
    for (int n = lane; n < nk; n += 32) l += expf(sm[L.s + h * cap + n] - m);
    l = warp_add(l);
    if (lane == 0) {
      sm[L.stat + h] = m;
      sm[L.stat + H + h] = l;
    }
  }
  if (CL > 1) cluster.sync(); else __syncthreads();
  for (int h = warp; h < H; h += kThreads / 32) {
    float m = -FLT_MAX, l = 0.f;
    for (int r = 0; r < CL; ++r) {
      const float* st = cluster.map_shared_rank(sm + L.stat, r);
      const float mr = st[h], lr = st[H + h];
      if (lr > 0.f) {
        const float mn = fmaxf(m, mr);
        l = l * expf(m - mn) + lr * expf(mr - mn);
        m = mn;
      }
    }
    const float inv = 1.0f / l;
    for (int n = lane; n < nk; n += 32) sm[L.s + h * cap + n] = expf(sm[L.s + h * cap + n] - m) * inv;
  }
  __syncthreads();

  // mixed weights
  const T* talk = static_cast<const T*>(p.talk);
  for (int item = tid; item < nk * H; item += kThreads) {
    const int h = item / nk, n = item - h * nk;
    float a = 0.f;
    for (int g = 0; g < H; ++g) a += to_f32(talk[h * H + g]) * sm[L.s + g * cap + n];
    sm[L.m + h * cap + n] = a;
  }
  __syncthreads();

  // values: a thread takes eight columns of a key head and every `groups`-th key
  const int vchunks = G * vp / 8;
  const int groups = vchunks < kThreads ? kThreads / vchunks : 1;
  const int grp = tid / vchunks;
  for (int r0 = 0; r0 < rep; r0 += kRep) {
    for (int vc0 = 0; vc0 < vchunks; vc0 += kThreads) {
      const int vc = vc0 + (groups > 1 ? tid - grp * vchunks : tid);
      const bool active = vc < vchunks && (groups == 1 || grp < groups);
      const int c = active ? vc / (vp / 8) : 0, d = active ? (vc - c * (vp / 8)) * 8 : 0;
      float acc[kRep][8] = {};
      if (active) {
        for (int n = groups > 1 ? grp : 0; n < nk; n += groups) {
          const int j = keys.position(n0 + n);
          const T* v = j >= pos0 ? new_v + (j - pos0) * p.ldp + static_cast<long long>(c) * vp + d
                                 : ring_v + (static_cast<long long>(window_slot(j, p.window, p.keep)) * G + c) * vp + d;
          float f[8];
          load8(v, f);
#pragma unroll
          for (int r = 0; r < kRep; ++r) {
            if (r0 + r < rep) {
              const float w = sm[L.m + (c * rep + r0 + r) * cap + n];
#pragma unroll
              for (int e = 0; e < 8; ++e) acc[r][e] += w * f[e];
            }
          }
        }
        float* red = sm + L.red + tid;      // [value][thread]: conflict-free
#pragma unroll
        for (int r = 0; r < kRep; ++r)
#pragma unroll
          for (int e = 0; e < 8; ++e) red[(r * 8 + e) * kThreads] = acc[r][e];
      }
      __syncthreads();
      if (vc < vchunks && (groups == 1 || grp == 0)) {
#pragma unroll
        for (int r = 0; r < kRep; ++r) {
          if (r0 + r >= rep) break;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float a = 0.f;
            for (int g = 0; g < groups; ++g) a += sm[L.red + (r * 8 + e) * kThreads + tid + g * vchunks];
            sm[L.o + (c * rep + r0 + r) * vp + d + e] = a;
          }
        }
      }
      __syncthreads();
    }
  }
  if (CL > 1) cluster.sync();
  T* out = static_cast<T*>(p.out) + row * p.ldo;
  for (int c = rank * kThreads + tid; c < H * vp; c += CL * kThreads) {
    float a = 0.f;
    for (int r = 0; r < CL; ++r) a += cluster.map_shared_rank(sm + L.o, r)[c];
    out[c] = from_f32<T>(a * p.out_scale);
  }
  if (CL > 1) cluster.sync();     // the other blocks read this block's shared memory until here
}

constexpr int kMaxDynSmem = 227 * 1024;

template <typename T>
cudaError_t launch_rows(const WindowAttnParams& p, cudaStream_t st) {
  const int n_max = p.keep + p.window;
  auto bytes = [&](int cl) {
    return static_cast<size_t>(rows_smem(p.H, p.dp, p.vp, (n_max + cl - 1) / cl).total) * sizeof(float);
  };
  // blocks per query: enough to fill the device when there are few queries, and enough for the
  // scores to fit in shared memory
  int cl = 1;
  const long long queries = static_cast<long long>(p.B) * p.S;
  while (cl < 8 && ((queries * cl < 148 && n_max / (2 * cl) >= 64) || bytes(cl) > kMaxDynSmem)) cl *= 2;
  if (bytes(cl) > kMaxDynSmem) return cudaErrorInvalidValue;
  auto kern = window_rows_kernel<T>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(static_cast<unsigned>(cl * p.S), static_cast<unsigned>(p.B), 1);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = bytes(cl);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cl;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, kern, p, (n_max + cl - 1) / cl);
}

}  // namespace

bool window_rows_supported(const WindowAttnParams& p) {
  return static_cast<size_t>(rows_smem(p.H, p.dp, p.vp, (p.keep + p.window + 7) / 8).total) * sizeof(float) <=
         kMaxDynSmem;
}

cudaError_t launch_head_norm(const WindowAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? head_norm_any<float>(p, st) : head_norm_any<bf16>(p, st);
}

cudaError_t launch_window_append(const WindowAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  const dim3 grid(p.S, p.B);
  return fp32 ? launch_kernel(window_append_kernel<float>, grid, dim3(128), 0, st, p)
              : launch_kernel(window_append_kernel<bf16>, grid, dim3(128), 0, st, p);
}

cudaError_t launch_window_rows(const WindowAttnParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_rows<float>(p, st) : launch_rows<bf16>(p, st);
}

}  // namespace cdeep

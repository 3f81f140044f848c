// Window attention of one new token per sequence (decoding), bound by the two passes over the ring.
// The heads' weights are mixed after the softmax, so the values cannot be weighted before the
// normalisers of all heads are known; three kernels:
//
//   scores   grid (splits, key heads x query-head groups, sequences): a block streams its share of the
//            keys of one key head for up to four query heads; 8 lanes share a key.  Scores (scaled,
//            biased) go to a workspace that stays in L2, with every block's softmax statistics.  The
//            block that holds the new token norms its key and writes key and value into the ring.
//   mix      grid (64 keys, sequences): combines the statistics, replaces the scores of all heads by
//            their mixed weights.
//   values   grid as for the scores, the splits of a (head group, sequence) form a thread-block
//            cluster: streams its share of the values; the parts are added through distributed shared
//            memory.
#include <cfloat>
#include <cooperative_groups.h>
#include "kernels.h"
#include "window_attention.cuh"

namespace cg = cooperative_groups;

namespace cdeep {

namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

struct DecodeParams {
  WindowAttnParams a;
  int splits;
  int n_max;        // keep + window
  float* scores;    // [B, H, n_max], then the mixed weights
  float* stats;     // [B, H, splits, 2]
};

struct KeyRange {
  int i, count, n0, nk;        // position of the query, its keys, this split's share
  int kept, first, slot0;      // keys n < kept: slot n; else slot0 + (n - kept), wrapped once
  int wrap;                    // slots from `wrap` on are lower by `window`
  int window;
  __device__ __forceinline__ KeyRange(const WindowAttnParams& p, int split, int splits) {
    i = window_pos0(p);
    const WindowKeys keys(i, p.window, p.keep);
    kept = keys.kept;
    first = keys.first;
    window = p.window;
    count = kept + (i - first + 1);
    const int chunk = (count + splits - 1) / splits;
    n0 = min(split * chunk, count);
    nk = min(chunk, count - n0);
    if (first < p.keep) {
      // the window still reaches kept positions: none of its slots has been used twice
      slot0 = first;
      wrap = 0x7fffffff;
    } else {
      slot0 = p.keep + (first - p.keep) % p.window;
      wrap = p.keep + p.window;
    }
  }
  __device__ __forceinline__ int slot(int n) const {
    if (n < kept) return n;
    const int s = slot0 + (n - kept);
    return s >= wrap ? s - window : s;
  }
  __device__ __forceinline__ int distance(int n) const { return n < kept ? i - n : i - first - (n - kept); }
};

__device__ __forceinline__ float group8_add(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}

// REP query heads per block; DC chunks of 8 elements per lane (head width up to 64 DC)
template <typename T, int REP, int DC>
__global__ void __launch_bounds__(kThreads, REP * DC <= 4 && sizeof(T) == 2 ? 3 : 1)
window_decode_scores_kernel(const DecodeParams p) {
  extern __shared__ float sm[];        // [REP][dp] queries
  __shared__ float s_m[kWarps][REP], s_l[kWarps][REP];
  pdl_enter();
  const WindowAttnParams& a = p.a;
  const int split = blockIdx.x, b = blockIdx.z, rep = a.H / a.G, groups = (rep + REP - 1) / REP;
  const int c = blockIdx.y / groups, h0 = c * rep + (blockIdx.y % groups) * REP;
  const int nh = min(REP, (c + 1) * rep - h0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane & 7, rg = lane >> 3;
  const int dp = a.dp, vp = a.vp;
  const KeyRange r(a, split, p.splits);
  const long long slots = a.keep + a.window;
  T* ring_k = static_cast<T*>(a.ring_k) + (b * slots * a.G + c) * dp;
  const long long stride = static_cast<long long>(a.G) * dp;
  const bool has_new = r.nk > 0 && r.n0 + r.nk == r.count;

  auto rms_scale = [&](const T* x) {
    float ss = 0.f;
    for (int d = lane; d < dp; d += 32) {
      const float f = to_f32(x[d]);
      ss += f * f;
    }
    return 1.0f / sqrtf(warp_add(ss) / static_cast<float>(a.dim) + a.eps);
  };
  for (int x = warp; x < nh; x += kWarps) {
    const T* q = static_cast<const T*>(a.q) + b * a.ldp + static_cast<long long>(h0 + x) * dp;
    const float s = rms_scale(q);
    for (int d = lane; d < dp; d += 32)
      sm[x * dp + d] = to_f32(from_f32<T>(to_f32(q[d]) * s * to_f32(static_cast<const T*>(a.q_w)[d]))) * a.scale;
  }
  if (has_new && warp == kWarps - 1) {
    // the new token's slot held a position that this query does not see
    const T* k = static_cast<const T*>(a.k) + b * a.ldp + static_cast<long long>(c) * dp;
    const float s = rms_scale(k);
    T* dst = ring_k + static_cast<long long>(r.slot(r.count - 1)) * stride;
    for (int d = lane; d < dp; d += 32) dst[d] = from_f32<T>(to_f32(k[d]) * s * to_f32(static_cast<const T*>(a.k_w)[d]));
  }
  if (has_new && warp == kWarps - 2) {
    const T* v = static_cast<const T*>(a.v) + b * a.ldp + static_cast<long long>(c) * vp;
    T* dst = static_cast<T*>(a.ring_v) + ((b * slots + r.slot(r.count - 1)) * a.G + c) * vp;
    for (int d = lane; d < vp; d += 32) dst[d] = v[d];
  }
  __syncthreads();
  float qf[REP][DC][8];
#pragma unroll
  for (int x = 0; x < REP; ++x)
#pragma unroll
    for (int e = 0; e < DC; ++e) {
      const int d = (e * 8 + sub) * 8;
#pragma unroll
      for (int y = 0; y < 8; ++y) qf[x][e][y] = (x < nh && d < dp) ? sm[x * dp + d + y] : 0.f;
    }
  // Rows in flight per lane.  The kAhead x REP scores of a lane group are finished by its lanes: lane
  // `sub` takes the head sub % REP and, in `kRounds` rounds, row sub / REP + round * (8 / REP).
  constexpr int kAhead = DC * sizeof(T) <= 4 ? 4 : 2;
  constexpr int kRowsRound = 8 / REP < kAhead ? 8 / REP : kAhead;
  constexpr int kRounds = kAhead / kRowsRound;
  constexpr int kStep = kWarps * 4;             // rows of the block per step
  const int my_head = sub % REP, my_row = sub / REP;
  float r1 = 0.f, r2 = 0.f, m = -FLT_MAX, l = 0.f;
  if (my_head < nh) {
    r1 = to_f32(static_cast<const T*>(a.r1)[h0 + my_head]);
    r2 = to_f32(static_cast<const T*>(a.r2)[h0 + my_head]);
  }
  float* out = p.scores + (static_cast<long long>(b) * a.H + h0 + (my_head < nh ? my_head : 0)) * p.n_max;
  for (int base = 0; base < r.nk; base += kStep * kAhead) {
    Raw8<T> kf[kAhead][DC];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      const int n = min(base + u * kStep + warp * 4 + rg, r.nk - 1);      // rows past the end are not used
      const T* k = ring_k + static_cast<long long>(r.slot(r.n0 + n)) * stride;
#pragma unroll
      for (int e = 0; e < DC; ++e) {
        const int d = (e * 8 + sub) * 8;
        raw_load(k + (d < dp ? d : 0), kf[u][e]);                         // past the head: the query is zero
      }
    }
    float s[kAhead][REP];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
#pragma unroll
      for (int x = 0; x < REP; ++x) s[u][x] = 0.f;
#pragma unroll
      for (int e = 0; e < DC; ++e) {
        float f[8];
        raw_unpack(kf[u][e], f);
#pragma unroll
        for (int x = 0; x < REP; ++x)
#pragma unroll
          for (int y = 0; y < 8; ++y) s[u][x] = fmaf(qf[x][e][y], f[y], s[u][x]);
      }
#pragma unroll
      for (int x = 0; x < REP; ++x) s[u][x] = group8_add(s[u][x]);
    }
#pragma unroll
    for (int y = 0; y < kRounds; ++y) {
      float v = 0.f;
#pragma unroll
      for (int u = 0; u < kRowsRound; ++u)
#pragma unroll
        for (int x = 0; x < REP; ++x) v = (my_row == u && my_head == x) ? s[y * kRowsRound + u][x] : v;
      const int n = base + (y * kRowsRound + my_row) * kStep + warp * 4 + rg;
      if (n < r.nk && my_head < nh && my_row < kRowsRound) {
        v -= r1 * score_log1p<T>(r2 * static_cast<float>(r.distance(r.n0 + n)));
        out[r.n0 + n] = v;
        const float mn = fmaxf(m, v);
        l = l * score_exp<T>(m - mn) + score_exp<T>(v - mn);
        m = mn;
      }
    }
  }
  // the block's statistics: the lanes of a head, then the warps
#pragma unroll
  for (int d = REP; d < 32; d <<= 1) {
    const float mo = __shfl_xor_sync(0xffffffffu, m, d), lo = __shfl_xor_sync(0xffffffffu, l, d);
    const float mn = fmaxf(m, mo);
    l = l * score_exp<T>(m - mn) + lo * score_exp<T>(mo - mn);
    m = mn;
  }
  if (lane < nh) {
    s_m[warp][lane] = m;
    s_l[warp][lane] = l;
  }
  __syncthreads();
  if (tid < nh) {
    m = s_m[0][tid];
    l = s_l[0][tid];
    for (int w = 1; w < kWarps; ++w) {
      const float mn = fmaxf(m, s_m[w][tid]);
      l = l * expf(m - mn) + s_l[w][tid] * expf(s_m[w][tid] - mn);
      m = mn;
    }
    float* st = p.stats + ((static_cast<long long>(b) * a.H + h0 + tid) * p.splits + split) * 2;
    st[0] = m;
    st[1] = l;
  }
}

constexpr int kMixKeys = 64;       // keys per block of the mixing kernel

template <typename T>
__global__ void __launch_bounds__(kThreads)
window_decode_mix_kernel(const DecodeParams p) {
  extern __shared__ float sm[];        // [H] maximum, [H] 1 / sum, [H][kMixKeys] weights
  pdl_enter();
  const WindowAttnParams& a = p.a;
  const int H = a.H, b = blockIdx.y, n0 = blockIdx.x * kMixKeys;
  const KeyRange r(a, 0, 1);
  const int n = min(kMixKeys, r.count - n0);
  if (n <= 0) return;
  for (int h = threadIdx.x; h < H; h += kThreads) {
    const float* st = p.stats + (static_cast<long long>(b) * H + h) * p.splits * 2;
    float m = -FLT_MAX, l = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      if (st[2 * s + 1] <= 0.f) continue;          // a split without keys
      const float mn = fmaxf(m, st[2 * s]);
      l = l * expf(m - mn) + st[2 * s + 1] * expf(st[2 * s] - mn);
      m = mn;
    }
    sm[h] = m;
    sm[H + h] = 1.0f / l;
  }
  __syncthreads();
  float* scores = p.scores + static_cast<long long>(b) * H * p.n_max + n0;
  float* w = sm + 2 * H;
  for (int x = threadIdx.x; x < H * kMixKeys; x += kThreads) {
    const int h = x / kMixKeys, k = x - h * kMixKeys;
    w[x] = k < n ? score_exp<T>(scores[static_cast<long long>(h) * p.n_max + k] - sm[h]) * sm[H + h] : 0.f;
  }
  __syncthreads();
  const T* talk = static_cast<const T*>(a.talk);
  for (int x = threadIdx.x; x < H * kMixKeys; x += kThreads) {
    const int h = x / kMixKeys, k = x - h * kMixKeys;
    float v = 0.f;
    for (int g = 0; g < H; ++g) v = fmaf(to_f32(talk[h * H + g]), w[g * kMixKeys + k], v);
    if (k < n) scores[static_cast<long long>(h) * p.n_max + k] = v;
  }
}

template <int REP>
__host__ __device__ inline int values_smem_floats(int vp) {
  return REP * 8 * kThreads + REP * vp;          // the threads' sums [REP * 8][kThreads], the block's output [REP][vp]
}

template <typename T, int REP>
__global__ void __launch_bounds__(kThreads, REP <= 2 && sizeof(T) == 2 ? 4 : 2)
window_decode_values_kernel(const DecodeParams p) {
  extern __shared__ float sm[];
  pdl_enter();
  cg::cluster_group cluster = cg::this_cluster();
  const WindowAttnParams& a = p.a;
  const int split = blockIdx.x, b = blockIdx.z, rep = a.H / a.G, groups = (rep + REP - 1) / REP;
  const int c = blockIdx.y / groups, h0 = c * rep + (blockIdx.y % groups) * REP;
  const int nh = min(REP, (c + 1) * rep - h0);
  const int tid = threadIdx.x, vp = a.vp;
  float* s_out = sm + REP * 8 * kThreads;
  const KeyRange r(a, split, p.splits);
  const long long slots = a.keep + a.window;
  const T* ring_v = static_cast<const T*>(a.ring_v) + (b * slots * a.G + c) * vp;
  const long long stride = static_cast<long long>(a.G) * vp;
  // a thread takes eight columns and every `rows`-th key
  const int cols = vp / 8, rows = kThreads / cols;               // vp <= 1024
  const int row = tid / cols, col = (tid - row * cols) * 8;
  const bool active = row < rows;
  const float* weights = p.scores + (static_cast<long long>(b) * a.H + h0) * p.n_max + r.n0;
  float acc[REP][8];
#pragma unroll
  for (int x = 0; x < REP; ++x)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[x][e] = 0.f;
  constexpr int kAhead = 4;
  if (active) {
    for (int at = row; at < r.nk; at += rows * kAhead) {
      Raw8<T> vf[kAhead];
      float w[kAhead][REP];
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        const int k = at + u * rows;
        const int kc = min(k, r.nk - 1);                         // past the end: weight zero
        raw_load(ring_v + static_cast<long long>(r.slot(r.n0 + kc)) * stride + col, vf[u]);
#pragma unroll
        for (int x = 0; x < REP; ++x)
          w[u][x] = k < r.nk && x < nh ? weights[static_cast<long long>(x) * p.n_max + k] : 0.f;
      }
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        float f[8];
        raw_unpack(vf[u], f);
#pragma unroll
        for (int x = 0; x < REP; ++x)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[x][e] = fmaf(w[u][x], f[e], acc[x][e]);
      }
    }
  }
#pragma unroll
  for (int x = 0; x < REP; ++x)
#pragma unroll
    for (int e = 0; e < 8; ++e) sm[(x * 8 + e) * kThreads + tid] = acc[x][e];
  __syncthreads();
  for (int idx = tid; idx < REP * vp; idx += kThreads) {
    const int x = idx / vp, d = idx - x * vp;
    const float* src = sm + (x * 8 + (d & 7)) * kThreads + (d >> 3);
    float v = 0.f;
    for (int y = 0; y < rows; ++y) v += src[y * cols];
    s_out[idx] = v;
  }
  if (p.splits > 1) cluster.sync(); else __syncthreads();
  T* out = static_cast<T*>(a.out) + b * a.ldo + static_cast<long long>(h0) * vp;
  for (int idx = split * kThreads + tid; idx < nh * vp; idx += p.splits * kThreads) {
    float v = 0.f;
    for (int s = 0; s < p.splits; ++s) v += cluster.map_shared_rank(s_out, s)[idx];
    out[idx] = from_f32<T>(v * a.out_scale);
  }
  if (p.splits > 1) cluster.sync();     // the other blocks read this block's shared memory until here
}

int choose_splits(const WindowAttnParams& a, int rep_block) {
  const int rep = a.H / a.G;
  const long long blocks = static_cast<long long>(a.B) * a.G * ((rep + rep_block - 1) / rep_block);
  int s = 1;
  while (s < 8 && blocks * s < 148 * 6 && (a.keep + a.window) / (2 * s) >= 64) s *= 2;
  return s;
}

int rep_block(const WindowAttnParams& a) {
  const int rep = a.H / a.G;
  return rep <= 1 ? 1 : rep <= 2 ? 2 : 4;
}

template <typename T, int REP, int DC>
cudaError_t launch_scores(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  return launch_kernel(window_decode_scores_kernel<T, REP, DC>, grid, dim3(kThreads), REP * p.a.dp * sizeof(float), st, p);
}

template <typename T, int REP>
cudaError_t launch_both(const DecodeParams& p, cudaStream_t st) {
  const int rep = p.a.H / p.a.G;
  const dim3 grid(p.splits, p.a.G * ((rep + REP - 1) / REP), p.a.B);
  cudaError_t e = p.a.dp <= 64    ? launch_scores<T, REP, 1>(p, grid, st)
                  : p.a.dp <= 128 ? launch_scores<T, REP, 2>(p, grid, st)
                                  : launch_scores<T, REP, 4>(p, grid, st);
  if (e != cudaSuccess) return e;
  const int mix_bytes = p.a.H * (2 + kMixKeys) * static_cast<int>(sizeof(float));
  e = cudaFuncSetAttribute(window_decode_mix_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, mix_bytes);
  if (e != cudaSuccess) return e;
  e = launch_kernel(window_decode_mix_kernel<T>, dim3((p.n_max + kMixKeys - 1) / kMixKeys, p.a.B), dim3(kThreads),
                    mix_bytes, st, p);
  if (e != cudaSuccess) return e;
  const int bytes = values_smem_floats<REP>(p.a.vp) * static_cast<int>(sizeof(float));
  auto kern = window_decode_values_kernel<T, REP>;
  e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = bytes;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = p.splits;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

template <typename T>
cudaError_t launch_typed(const DecodeParams& p, cudaStream_t st) {
  switch (rep_block(p.a)) {
    case 1: return launch_both<T, 1>(p, st);
    case 2: return launch_both<T, 2>(p, st);
    default: return launch_both<T, 4>(p, st);
  }
}

}  // namespace

bool window_decode_supported(const WindowAttnParams& a) {
  return a.dp <= 256 && a.vp <= 1024 && a.H <= 256 && a.G * ((a.H / a.G + 3) / 4) <= 65535;
}

size_t window_decode_workspace_bytes(const WindowAttnParams& a) {
  return static_cast<size_t>(a.B) * a.H * (a.keep + a.window + 2 * choose_splits(a, rep_block(a))) * sizeof(float);
}

cudaError_t launch_window_decode(const WindowAttnParams& a, void* ws, int fp32, cudaStream_t st) {
  if (a.B == 0) return cudaSuccess;
  DecodeParams p;
  p.a = a;
  p.splits = choose_splits(a, rep_block(a));
  p.n_max = a.keep + a.window;
  p.scores = static_cast<float*>(ws);
  p.stats = p.scores + static_cast<size_t>(a.B) * a.H * p.n_max;
  return fp32 ? launch_typed<float>(p, st) : launch_typed<bf16>(p, st);
}

}  // namespace cdeep

// Latent attention of a few new tokens in bf16 without expanding the latent: one cached row serves all
// heads of its sequence, so the cache is read once per tile of query rows.
//
//   latent_absorb_kernel   q~_h = uk_h^T q_h next to the rotated part: rows [B * S, H, rankp + rotp]
//   latent_attend_kernel   scores against the cached rows, online softmax, weighted latent; the keys of a
//                          sequence are dealt to `splits` blocks, which leave fp32 partial results
//   latent_finish_kernel   sum over the splits, uv_h, gate
//
// Query rows of a sequence are its (token, head) pairs, 16 or 32 to a block; warp-level products, since
// 16 heads fill one m16 tile where a 128-row tensor-memory tile would be mostly padding.
#include "kernels.h"
#include "latent_attention.cuh"
#include "mma.cuh"

namespace cdeep {

namespace {

constexpr int kThreads = 256;
constexpr int kKeys = 64;        // keys per tile
constexpr int kLdS = kKeys + 4;
constexpr int kLdP = kKeys + 8;
constexpr int kMaxSplits = 32;

struct DecodeParams {
  LatentParams a;
  bf16* q;             // [B * S, H, W]
  float* o;            // [B, splits, S * H, rankp]
  float* ml;           // [B, splits, S * H, 2]: running maximum (log2 domain) and sum
  int splits;
};

// ---------------------------------------------------------------- q to the latent's space
// 64 rows x 64 columns per block; warp w: rows (w & 3) * 16, columns (w >> 2) * 32
__global__ void __launch_bounds__(kThreads)
latent_absorb_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const LatentParams& a = p.a;
  const int n0 = blockIdx.x * 64, h = blockIdx.y, m0 = blockIdx.z * 64, rows = a.B * a.S;
  const int ld = a.dimp + 8, W = a.rankp + a.rotp, per = a.dimp / 8;
  bf16* sa = reinterpret_cast<bf16*>(smem);
  bf16* sb = sa + 64 * ld;
  const bf16* q = static_cast<const bf16*>(a.q) + static_cast<long long>(h) * (a.dimp + a.rotp);
  const bf16* w = static_cast<const bf16*>(a.uk_t) + static_cast<long long>(h) * a.rankp * a.dimp;
  for (int i = threadIdx.x; i < 64 * per; i += kThreads) {
    const int r = i / per, c = (i - r * per) * 8;
    if (m0 + r < rows) copy16_async(sa + r * ld + c, q + (m0 + r) * a.ldp + c);
    else *reinterpret_cast<uint4*>(sa + r * ld + c) = make_uint4(0, 0, 0, 0);
    if (n0 + r < a.rankp) copy16_async(sb + r * ld + c, w + static_cast<long long>(n0 + r) * a.dimp + c);
    else *reinterpret_cast<uint4*>(sb + r * ld + c) = make_uint4(0, 0, 0, 0);
  }
  copy_commit();
  if (n0 == 0) {                       // the rotated part moves along
    const int pr = a.rotp / 8;
    for (int i = threadIdx.x; i < 64 * pr; i += kThreads) {
      const int r = i / pr, c = (i - r * pr) * 8;
      if (m0 + r < rows)
        *reinterpret_cast<uint4*>(p.q + (static_cast<long long>(m0 + r) * a.H + h) * W + a.rankp + c) =
            *reinterpret_cast<const uint4*>(q + (m0 + r) * a.ldp + a.dimp + c);
    }
  }
  copy_wait<0>();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int mr = (warp & 3) * 16, nc = (warp >> 2) * 32;
  if (m0 + mr >= rows || n0 + nc >= a.rankp) return;
  float acc[4][4] = {};
  for (int d = 0; d < a.dimp; d += 16) {
    uint32_t fa[4];
    ldsm4(fa, smem_addr(sa + (mr + (lane & 15)) * ld + d + (lane >> 4) * 8));
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      uint32_t fb[4];
      ldsm4(fb, smem_addr(sb + (nc + x * 16 + (lane & 7) + ((lane >> 4) << 3)) * ld + d + ((lane >> 3) & 1) * 8));
      mma16816(acc[2 * x], fa, fb[0], fb[1]);
      mma16816(acc[2 * x + 1], fa, fb[2], fb[3]);
    }
  }
#pragma unroll
  for (int x = 0; x < 4; ++x) {
    const int col = n0 + nc + x * 8 + (lane & 3) * 2;
    if (n0 + nc + x * 8 >= a.rankp) continue;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = m0 + mr + (lane >> 2) + r * 8;
      if (row < rows)
        *reinterpret_cast<uint32_t*>(p.q + (static_cast<long long>(row) * a.H + h) * W + col) =
            bf_pack(acc[x][2 * r], acc[x][2 * r + 1]);
    }
  }
}

// ---------------------------------------------------------------- attention over the cached rows
struct AttendSmem {     // byte offsets
  int q, k, s, p, alpha, total;
};
__host__ __device__ inline AttendSmem attend_smem(int W, int mt) {
  AttendSmem s;
  s.q = 0;
  s.k = s.q + 16 * mt * (W + 8) * 2;
  s.s = s.k + 2 * kKeys * (W + 8) * 2;
  s.p = s.s + 2 * 16 * mt * kLdS * 4;
  s.alpha = s.p + 16 * mt * kLdP * 2;
  s.total = s.alpha + 16 * mt * 4;
  return s;
}

// MT row tiles of 16; PP: pairs of 8 latent columns per warp (rankp <= 128 PP)
template <int MT, int PP>
__global__ void __launch_bounds__(kThreads, 1)
latent_attend_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const LatentParams& a = p.a;
  constexpr int M = 16 * MT;
  const int split = blockIdx.x, r0 = blockIdx.y * M, b = blockIdx.z;
  const int R = a.S * a.H, W = a.rankp + a.rotp, ld = W + 8, per = W / 8;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const AttendSmem off = attend_smem(W, MT);
  bf16* sq = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sk = reinterpret_cast<bf16*>(smem + off.k);
  float* ss = reinterpret_cast<float*>(smem + off.s);
  bf16* sp = reinterpret_cast<bf16*>(smem + off.p);
  float* s_alpha = reinterpret_cast<float*>(smem + off.alpha);
  const int pos0 = first_position(a);
  const int len = min(pos0 + (min(r0 + M, R) - 1) / a.H + 1, a.capacity);     // keys that any row of the tile sees
  const int tiles = (len + kKeys - 1) / kKeys;
  const int t_lo = static_cast<int>(static_cast<long long>(tiles) * split / p.splits);
  const int t_hi = static_cast<int>(static_cast<long long>(tiles) * (split + 1) / p.splits);
  const bf16* cache = static_cast<const bf16*>(a.cache) + static_cast<long long>(b) * a.capacity * W;
  const bf16* q = p.q + (static_cast<long long>(b) * R + r0) * W;

  auto fetch = [&](int tile) {
    bf16* dst = sk + (tile & 1) * kKeys * ld;
    const int j0 = tile * kKeys;
    // a warp copies whole rows, eight of them
    for (int r = warp; r < kKeys; r += kThreads / 32) {
      const bool ok = j0 + r < len;
      const bf16* src = cache + static_cast<long long>(j0 + r) * W;
      for (int c = lane; c < per; c += 32) {
        if (ok) copy16_async(dst + r * ld + c * 8, src + c * 8);
        else *reinterpret_cast<uint4*>(dst + r * ld + c * 8) = make_uint4(0, 0, 0, 0);
      }
    }
  };
  for (int i = threadIdx.x; i < M * per; i += kThreads) {
    const int r = i / per, c = (i - r * per) * 8;
    if (r0 + r < R) copy16_async(sq + r * ld + c, q + static_cast<long long>(r) * W + c);
    else *reinterpret_cast<uint4*>(sq + r * ld + c) = make_uint4(0, 0, 0, 0);
  }
  if (t_lo < t_hi) fetch(t_lo);
  copy_commit();

  // softmax state of the rows warp * 2 MT + x (a warp owns whole rows there)
  float m_run[2 * MT], l_run[2 * MT];
#pragma unroll
  for (int x = 0; x < 2 * MT; ++x) {
    m_run[x] = -INFINITY;
    l_run[x] = 0.f;
  }
  float acc[MT][PP][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int x = 0; x < PP; ++x)
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[m][x][y][e] = 0.f;
  const float scale2 = a.scale * 1.4426950408889634f;
  const int kg = (warp & 3) * 16, half = warp >> 2;
  const int steps = W / 16, d_lo = half ? (steps + 1) / 2 : 0, d_hi = half ? steps : (steps + 1) / 2;

  for (int tile = t_lo; tile < t_hi; ++tile) {
    if (tile + 1 < t_hi) fetch(tile + 1);
    copy_commit();
    copy_wait<1>();
    __syncthreads();
    const bf16* k = sk + (tile & 1) * kKeys * ld;
    // ---- scores: 16 keys per warp, half of the depth
    {
      float s[MT][2][4] = {};
#pragma unroll 4
      for (int d = d_lo; d < d_hi; ++d) {
        uint32_t fb[4];
        ldsm4(fb, smem_addr(k + (kg + (lane & 7) + ((lane >> 4) << 3)) * ld + d * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t fa[4];
          ldsm4(fa, smem_addr(sq + (m * 16 + (lane & 15)) * ld + d * 16 + (lane >> 4) * 8));
          mma16816(s[m][0], fa, fb[0], fb[1]);
          mma16816(s[m][1], fa, fb[2], fb[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
          for (int r = 0; r < 2; ++r)
            *reinterpret_cast<float2*>(ss + (half * M + m * 16 + (lane >> 2) + r * 8) * kLdS + kg + y * 8 + (lane & 3) * 2) =
                make_float2(s[m][y][2 * r], s[m][y][2 * r + 1]);
    }
    __syncthreads();
    // ---- softmax: 2 MT rows per warp, two keys per lane
#pragma unroll
    for (int x = 0; x < 2 * MT; ++x) {
      const int row = warp * 2 * MT + x;
      const int vis = pos0 + (r0 + row) / a.H - tile * kKeys;           // last visible key of the tile
      const float2 u = *reinterpret_cast<const float2*>(ss + row * kLdS + lane * 2);
      const float2 v = *reinterpret_cast<const float2*>(ss + (M + row) * kLdS + lane * 2);
      const float s0 = lane * 2 <= vis ? (u.x + v.x) * scale2 : -INFINITY;
      const float s1 = lane * 2 + 1 <= vis ? (u.y + v.y) * scale2 : -INFINITY;
      const float m_new = fmaxf(m_run[x], warp_max(fmaxf(s0, s1)));
      const float m_safe = m_new == -INFINITY ? 0.f : m_new;            // no visible key so far
      const float alpha = exp2_approx(m_run[x] - m_safe);
      const float e0 = exp2_approx(s0 - m_safe), e1 = exp2_approx(s1 - m_safe);
      l_run[x] = l_run[x] * alpha + warp_add(e0 + e1);
      m_run[x] = m_new;
      *reinterpret_cast<uint32_t*>(sp + row * kLdP + lane * 2) = bf_pack(e0, e1);
      if (lane == 0) s_alpha[row] = alpha;
    }
    __syncthreads();
    // ---- weighted latent: this warp's columns
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = s_alpha[m * 16 + (lane >> 2)], f1 = s_alpha[m * 16 + (lane >> 2) + 8];
      if (f0 != 1.f || f1 != 1.f) {
#pragma unroll
        for (int x = 0; x < PP; ++x)
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            acc[m][x][y][0] *= f0;
            acc[m][x][y][1] *= f0;
            acc[m][x][y][2] *= f1;
            acc[m][x][y][3] *= f1;
          }
      }
    }
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      uint32_t fp[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4(fp[m], smem_addr(sp + (m * 16 + (lane & 15)) * kLdP + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int x = 0; x < PP; ++x) {
        const int col = (warp + 8 * x) * 16;
        if (col < a.rankp) {
          uint32_t fb[4];
          ldsm4_t(fb, smem_addr(k + (kk * 16 + (lane & 15)) * ld + col + (lane >> 4) * 8));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma16816(acc[m][x][0], fp[m], fb[0], fb[1]);
            mma16816(acc[m][x][1], fp[m], fb[2], fb[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  copy_wait<0>();
  const long long base = (static_cast<long long>(b) * p.splits + split) * R + r0;
#pragma unroll
  for (int x = 0; x < 2 * MT; ++x) {
    const int row = warp * 2 * MT + x;
    if (lane == 0 && r0 + row < R) {
      p.ml[(base + row) * 2] = m_run[x];
      p.ml[(base + row) * 2 + 1] = l_run[x];
    }
  }
  if (t_lo >= t_hi) return;            // nothing of this split: its sum is zero and its rows are not read
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int x = 0; x < PP; ++x) {
      const int col = (warp + 8 * x) * 16;
      if (col >= a.rankp) continue;
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int row = m * 16 + (lane >> 2) + r * 8;
          if (r0 + row < R)
            *reinterpret_cast<float2*>(p.o + (base + row) * a.rankp + col + y * 8 + (lane & 3) * 2) =
                make_float2(acc[m][x][y][2 * r], acc[m][x][y][2 * r + 1]);
        }
    }
}

// ---------------------------------------------------------------- splits, uv, gate
// 16 tokens of one head and 64 value columns per block, eight of them per warp
__global__ void __launch_bounds__(kThreads)
latent_finish_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_w[16][kMaxSplits];
  pdl_enter();
  const LatentParams& a = p.a;
  const int n0 = blockIdx.x * 64, h = blockIdx.y, m0 = blockIdx.z * 16, rows = a.B * a.S;
  const int R = a.S * a.H, ld = a.rankp + 8, per = a.rankp / 8;
  bf16* sa = reinterpret_cast<bf16*>(smem);        // [16][ld]
  bf16* sb = sa + 16 * ld;                         // [64][ld]
  const bf16* uv = static_cast<const bf16*>(a.uv) + (static_cast<long long>(h) * a.vp + n0) * a.rankp;
  for (int i = threadIdx.x; i < 64 * per; i += kThreads) {
    const int r = i / per, c = (i - r * per) * 8;
    if (n0 + r < a.vp) copy16_async(sb + r * ld + c, uv + static_cast<long long>(r) * a.rankp + c);
    else *reinterpret_cast<uint4*>(sb + r * ld + c) = make_uint4(0, 0, 0, 0);
  }
  copy_commit();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  // weights of the splits: two rows per warp, a split per lane
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int i = warp * 2 + x, row = m0 + i;
    float m = -INFINITY, l = 0.f;
    if (row < rows && lane < p.splits) {
      const int b = row / a.S, t = row - b * a.S;
      const float2 v = *reinterpret_cast<const float2*>(
          p.ml + ((static_cast<long long>(b) * p.splits + lane) * R + t * a.H + h) * 2);
      m = v.x;
      l = v.y;
    }
    const float top = warp_max(m);
    const float f = l > 0.f ? exp2_approx(m - top) : 0.f;
    const float sum = warp_add(l * f);
    if (lane < p.splits) s_w[i][lane] = sum > 0.f ? f / sum : 0.f;
  }
  __syncthreads();
#pragma unroll 2
  for (int i = threadIdx.x; i < 16 * per; i += kThreads) {
    const int r = i / per, c = (i - r * per) * 8, row = m0 + r;
    float o[8] = {};
    if (row < rows) {
      const int b = row / a.S, t = row - b * a.S;
      const float* src = p.o + (static_cast<long long>(b) * p.splits * R + t * a.H + h) * a.rankp + c;
      for (int s0 = 0; s0 < p.splits; s0 += 4) {
        float w[4], f[4][8];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          w[x] = s0 + x < p.splits ? s_w[r][s0 + x] : 0.f;   // zero: the split has no rows to read
          if (w[x] != 0.f) load8(src + static_cast<long long>(s0 + x) * R * a.rankp, f[x]);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (w[x] != 0.f) {
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = fmaf(w[x], f[x][e], o[e]);
          }
      }
    }
    store8(sa + r * ld + c, o);
  }
  copy_wait<0>();
  __syncthreads();
  const int nc = warp * 8;
  if (n0 + nc >= a.vp) return;
  float acc[4] = {};
  for (int d = 0; d < a.rankp; d += 16) {
    uint32_t fa[4], fb[4];
    ldsm4(fa, smem_addr(sa + (lane & 15) * ld + d + (lane >> 4) * 8));
    ldsm4(fb, smem_addr(sb + (nc + (lane & 7)) * ld + d + ((lane >> 3) & 1) * 8));
    mma16816(acc, fa, fb[0], fb[1]);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = m0 + (lane >> 2) + r * 8;
    if (row >= rows) continue;
    const float g = a.out_scale * sigmoid_precise(to_f32(static_cast<const bf16*>(a.gate)[row * a.ldp + h]));
    *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + row * a.ldo + static_cast<long long>(h) * a.vp + n0 + nc +
                                 (lane & 3) * 2) = bf_pack(acc[2 * r] * g, acc[2 * r + 1] * g);
  }
}

constexpr int kMaxSmem = 227 * 1024;

int row_tiles(const LatentParams& a, int mt) { return (a.S * a.H + 16 * mt - 1) / (16 * mt); }
int pick_mt(const LatentParams& a) {
  return a.S * a.H > 16 && attend_smem(a.rankp + a.rotp, 2).total <= kMaxSmem ? 2 : 1;
}

// Key ranges per row tile: fewest rounds of blocks (one block per SM), counting about one and a half
// tiles per block for its start and end.
int pick_splits(const LatentParams& a) {
  const int sms = current_sm_count();
  const int len = a.pos_dev ? a.capacity : a.pos0 + a.S, tiles = (len + kKeys - 1) / kKeys;
  const long long blocks = static_cast<long long>(a.B) * row_tiles(a, pick_mt(a));
  int best = 1;
  long long cost = -1;
  for (int s = 1; s <= kMaxSplits && s <= tiles; ++s) {
    const long long c = (blocks * s + sms - 1) / sms * (2 * ((tiles + s - 1) / s) + 3);
    if (cost < 0 || c < cost) {
      cost = c;
      best = s;
    }
  }
  return best;
}

size_t align256(size_t n) { return (n + 255) & ~static_cast<size_t>(255); }

template <int MT, int PP>
cudaError_t launch_attend(const DecodeParams& p, cudaStream_t st) {
  const int bytes = attend_smem(p.a.rankp + p.a.rotp, MT).total;
  auto kern = latent_attend_kernel<MT, PP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  return launch_kernel(kern, dim3(p.splits, row_tiles(p.a, MT), p.a.B), dim3(kThreads), bytes, st, p);
}

}  // namespace

bool latent_decode_supported(const LatentParams& a) {
  return a.rankp <= 512 && a.dimp <= 512 && attend_smem(a.rankp + a.rotp, 1).total <= kMaxSmem && a.H <= 65535 &&
         static_cast<long long>(a.S) * a.H <= 65535 * 16 && static_cast<long long>(a.B) * a.S <= 65535 * 16;
}

size_t latent_decode_workspace_bytes(const LatentParams& a) {
  const size_t rows = static_cast<size_t>(a.B) * a.S * a.H, splits = pick_splits(a);
  return align256(rows * (a.rankp + a.rotp) * 2) + align256(rows * splits * a.rankp * 4) + rows * splits * 8;
}

cudaError_t launch_latent_decode(const LatentParams& a, void* ws, cudaStream_t st) {
  if (a.B == 0 || a.S == 0) return cudaSuccess;
  DecodeParams p;
  p.a = a;
  p.splits = pick_splits(a);
  const size_t rows = static_cast<size_t>(a.B) * a.S * a.H;
  char* at = static_cast<char*>(ws);
  p.q = reinterpret_cast<bf16*>(at);
  at += align256(rows * (a.rankp + a.rotp) * 2);
  p.o = reinterpret_cast<float*>(at);
  at += align256(rows * p.splits * a.rankp * 4);
  p.ml = reinterpret_cast<float*>(at);
  const int tokens = a.B * a.S;
  const int absorb = 2 * 64 * (a.dimp + 8) * 2, finish = 80 * (a.rankp + 8) * 2;
  cudaError_t e = cudaFuncSetAttribute(latent_absorb_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, absorb);
  if (e != cudaSuccess) return e;
  e = cudaFuncSetAttribute(latent_finish_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, finish);
  if (e != cudaSuccess) return e;
  e = launch_kernel(latent_absorb_kernel, dim3((a.rankp + 63) / 64, a.H, (tokens + 63) / 64), dim3(kThreads), absorb, st, p);
  if (e != cudaSuccess) return e;
  const int mt = pick_mt(a);
  if (mt == 1)
    e = a.rankp <= 128 ? launch_attend<1, 1>(p, st) : a.rankp <= 256 ? launch_attend<1, 2>(p, st) : launch_attend<1, 4>(p, st);
  else
    e = a.rankp <= 128 ? launch_attend<2, 1>(p, st) : a.rankp <= 256 ? launch_attend<2, 2>(p, st) : launch_attend<2, 4>(p, st);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_finish_kernel, dim3((a.vp + 63) / 64, a.H, (tokens + 15) / 16), dim3(kThreads), finish, st, p);
}

}  // namespace cdeep

// Latent attention of a few new tokens in bf16 without expanding the latent: one cached row serves all
// heads of its sequence, so the cache is read once per tile of query rows.
//
//   latent_absorb_kernel   q~_h = uk_h^T q_h next to the rotated part: rows [B * S, H, rankp + rotp]
//   latent_attend_kernel   scores against the cached rows, online softmax, weighted latent; the keys of a
//                          sequence are dealt to `splits` blocks, which leave fp32 partial results
//   latent_finish_kernel   sum over the splits, uv_h, gate
//
// Query rows of a sequence are its (token, head) pairs, 16 or 32 to a block; warp-level products, since
// 16 heads fill one m16 tile where a 128-row tensor-memory tile would be mostly padding.  Cached rows
// arrive by one bulk copy each, several tiles ahead.
#include "kernels.h"
#include "latent_attention.cuh"
#include "mma.cuh"
#include "ptx.cuh"

namespace cdeep {

namespace {

constexpr int kThreads = 256;
constexpr int kKeys = 32;        // keys per tile
constexpr int kLdS = kKeys + 4;
constexpr int kWarps = 8;        // of the attention kernel
constexpr int kParts = kWarps / 2;   // the depth of a score is dealt to as many warps
constexpr int kMaxStages = 4;    // tiles in flight
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
  int q, k, s, p, alpha, bars, stages, total;
};
constexpr int kMaxSmem = 227 * 1024;
constexpr int kHalfSmem = 113 * 1024;    // two blocks per SM
__host__ __device__ inline AttendSmem attend_smem(int W, int mt) {
  AttendSmem s;
  const int stage = kKeys * (W + 8) * 2;
  s.q = 0;
  s.s = s.q + 16 * mt * (W + 8) * 2;
  s.p = s.s + kParts * 16 * mt * kLdS * 4;
  s.alpha = s.p + 16 * mt * kLdP * 2;
  s.bars = s.alpha + 16 * mt * 4;
  s.k = s.bars + (kMaxStages + 2) * 8;
  // two blocks per SM that work in turn when two stages leave room for it, else one with more in flight
  s.stages = (kHalfSmem - s.k) / stage;
  if (s.stages < 2) s.stages = (kMaxSmem - s.k) / stage;
  if (s.stages > kMaxStages) s.stages = kMaxStages;
  s.total = s.k + s.stages * stage;
  return s;
}

// one row of `bytes` (a multiple of 16; both addresses 16-byte aligned), completing on `bar`
__device__ __forceinline__ void bulk_copy(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                   smem_addr(dst)), "l"(src), "r"(bytes), "r"(smem_addr(bar))
               : "memory");
}

// MT row tiles of 16; PP: pairs of 8 latent columns per warp (rankp <= 128 PP)
template <int MT, int PP>
__global__ void __launch_bounds__(kWarps * 32, MT == 1 ? 2 : 1)
latent_attend_kernel(const DecodeParams p, int* status) {
  extern __shared__ __align__(16) unsigned char smem[];
  const LatentParams& a = p.a;
  constexpr int M = 16 * MT, kRows = M / kWarps;      // rows whose softmax a warp owns
  const int split = blockIdx.x, r0 = blockIdx.y * M, b = blockIdx.z;
  const int R = a.S * a.H, W = a.rankp + a.rotp, ld = W + 8, per = W / 8;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const AttendSmem off = attend_smem(W, MT);
  bf16* sq = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sk = reinterpret_cast<bf16*>(smem + off.k);
  float* ss = reinterpret_cast<float*>(smem + off.s);
  bf16* sp = reinterpret_cast<bf16*>(smem + off.p);
  float* s_alpha = reinterpret_cast<float*>(smem + off.alpha);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + off.bars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + kMaxStages);
  if (threadIdx.x == 0) {
    for (int i = 0; i < off.stages; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  pdl_enter();
  __syncthreads();
  const int pos0 = first_position(a);
  const int len = min(pos0 + (min(r0 + M, R) - 1) / a.H + 1, a.capacity);     // keys that any row of the tile sees
  const int tiles = (len + kKeys - 1) / kKeys;
  const int t_lo = static_cast<int>(static_cast<long long>(tiles) * split / p.splits);
  const int t_hi = static_cast<int>(static_cast<long long>(tiles) * (split + 1) / p.splits);
  const bf16* cache = static_cast<const bf16*>(a.cache) + static_cast<long long>(b) * a.capacity * W;
  const bf16* q = p.q + (static_cast<long long>(b) * R + r0) * W;

  // four rows of the tile per warp, one per lane (a warp's copies are issued one after the other); rows
  // beyond the sequence are zeroed (a weight of zero must not meet what an earlier kernel left there)
  constexpr int kPerWarp = kKeys / kWarps;
  auto fetch = [&](int tile, int stage) {
    if (lane >= kPerWarp) return;
    const int j0 = tile * kKeys, rows = min(kKeys, len - j0), row = warp * kPerWarp + lane;
    bf16* dst = sk + (stage * kKeys + row) * ld;
    if (row == 0) mbar_arrive_expect_tx(&full[stage], static_cast<uint32_t>(rows * W * 2));
    if (row < rows) bulk_copy(dst, cache + static_cast<long long>(j0 + row) * W, W * 2, &full[stage]);
    else
      for (int c = 0; c < W; c += 8) *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
  };
  for (int x = 0; x < off.stages && t_lo + x < t_hi; ++x) fetch(t_lo + x, x);
  for (int i = threadIdx.x; i < M * per; i += kWarps * 32) {
    const int r = i / per, c = (i - r * per) * 8;
    if (r0 + r < R) copy16_async(sq + r * ld + c, q + static_cast<long long>(r) * W + c);
    else *reinterpret_cast<uint4*>(sq + r * ld + c) = make_uint4(0, 0, 0, 0);
  }
  copy_commit();

  // softmax state of the rows warp * 2 MT + x (a warp owns whole rows there)
  float m_run[kRows], l_run[kRows];
#pragma unroll
  for (int x = 0; x < kRows; ++x) {
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
  const int kg = (warp & 1) * 16, part = warp >> 1;
  const int steps = W / 16, d_lo = steps * part / kParts, d_hi = steps * (part + 1) / kParts;

  // partial scores of a tile: 16 keys and a part of the depth per warp
  auto scores = [&](int stage, uint32_t phase) {
    mbar_wait(&full[stage], phase, abort_flag);
    const bf16* k = sk + stage * kKeys * ld;
    float s[MT][2][4] = {};
#pragma unroll 3
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
          *reinterpret_cast<float2*>(ss + (part * M + m * 16 + (lane >> 2) + r * 8) * kLdS + kg + y * 8 + (lane & 3) * 2) =
              make_float2(s[m][y][2 * r], s[m][y][2 * r + 1]);
  };

  copy_wait<0>();
  __syncthreads();
  if (t_lo < t_hi) scores(0, 0);
  __syncthreads();
  int stage = 0;
  uint32_t phase = 0;
  for (int tile = t_lo; tile < t_hi; ++tile) {
    // ---- softmax: kRows rows per warp, a key per lane
#pragma unroll
    for (int x = 0; x < kRows; ++x) {
      const int row = warp * kRows + x;
      const int vis = pos0 + (r0 + row) / a.H - tile * kKeys;           // last visible key of the tile
      float s = 0.f;
#pragma unroll
      for (int y = 0; y < kParts; ++y) s += ss[(y * M + row) * kLdS + lane];
      s = lane <= vis ? s * scale2 : -INFINITY;
      const float m_new = fmaxf(m_run[x], warp_max(s));
      const float m_safe = m_new == -INFINITY ? 0.f : m_new;            // no visible key so far
      const float alpha = exp2_approx(m_run[x] - m_safe);
      const float e = exp2_approx(s - m_safe);
      l_run[x] = l_run[x] * alpha + e;                                  // this lane's keys
      m_run[x] = m_new;
      sp[row * kLdP + lane] = __float2bfloat16_rn(e);
      if (lane == 0) s_alpha[row] = alpha;
    }
    __syncthreads();
    // ---- weighted latent: this warp's columns; then the next tile's scores
    const bf16* k = sk + stage * kKeys * ld;
    const int next = stage + 1 == off.stages ? 0 : stage + 1;
    const uint32_t next_phase = next ? phase : phase ^ 1u;
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
        const int col = (warp + kWarps * x) * 16;
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
    if (tile + 1 < t_hi) scores(next, next_phase);
    __syncthreads();
    if (tile + off.stages < t_hi) fetch(tile + off.stages, stage);
    stage = next;
    phase = next_phase;
  }
  if (threadIdx.x == 0 && *abort_flag) atomicExch(status, 1);
  const long long base = (static_cast<long long>(b) * p.splits + split) * R + r0;
#pragma unroll
  for (int x = 0; x < kRows; ++x) {
    const int row = warp * kRows + x;
    const float l = warp_add(l_run[x]);
    if (lane == 0 && r0 + row < R) {
      p.ml[(base + row) * 2] = m_run[x];
      p.ml[(base + row) * 2 + 1] = l;
    }
  }
  if (t_lo >= t_hi) return;            // nothing of this split: its sum is zero and its rows are not read
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int x = 0; x < PP; ++x) {
      const int col = (warp + kWarps * x) * 16;
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
constexpr int kValueCols = 32;   // value columns per block of the last kernel

// 16 tokens of one head and 32 value columns per block; warp w: columns (w & 3) * 8, half of the depth
__global__ void __launch_bounds__(kThreads)
latent_finish_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_w[16][kMaxSplits];
  __shared__ float s_half[16][kValueCols + 2];
  pdl_enter();
  const LatentParams& a = p.a;
  const int n0 = blockIdx.x * kValueCols, h = blockIdx.y, m0 = blockIdx.z * 16, rows = a.B * a.S;
  const int R = a.S * a.H, ld = a.rankp + 8;
  bf16* sa = reinterpret_cast<bf16*>(smem);        // [16][ld]
  bf16* sb = sa + 16 * ld;                         // [kValueCols][ld]
  const bf16* uv = static_cast<const bf16*>(a.uv) + (static_cast<long long>(h) * a.vp + n0) * a.rankp;
  {
    const int r = threadIdx.x / (kThreads / kValueCols);
    for (int c = threadIdx.x % (kThreads / kValueCols) * 8; c < a.rankp; c += kThreads / kValueCols * 8) {
      if (n0 + r < a.vp) copy16_async(sb + r * ld + c, uv + r * a.rankp + c);
      else *reinterpret_cast<uint4*>(sb + r * ld + c) = make_uint4(0, 0, 0, 0);
    }
  }
  copy_commit();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float g[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = m0 + (lane >> 2) + r * 8;
    g[r] = row < rows ? to_f32(static_cast<const bf16*>(a.gate)[row * a.ldp + h]) : 0.f;
  }
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
  // sixteen threads per row, up to four pieces of eight elements each.  Every load is made, all in flight
  // together: what a split without rows left in the workspace is replaced by zero afterwards.
  {
    constexpr int kItems = 4;
    const int i = threadIdx.x >> 4, row = min(m0 + i, rows - 1), c0 = (threadIdx.x & 15) * 8;
    const int b = row / a.S, t = row - b * a.S;
    const float* src = p.o + (static_cast<long long>(b) * p.splits * R + t * a.H + h) * a.rankp;
    int at[kItems];
#pragma unroll
    for (int x = 0; x < kItems; ++x) at[x] = c0 + x * 128 < a.rankp ? c0 + x * 128 : 0;
    float o[kItems][8] = {};
#pragma unroll 2
    for (int s = 0; s < p.splits; ++s, src += static_cast<long long>(R) * a.rankp) {
      const float w = s_w[i][s];
      float f[kItems][8];
#pragma unroll
      for (int x = 0; x < kItems; ++x) load8(src + at[x], f[x]);
#pragma unroll
      for (int x = 0; x < kItems; ++x)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[x][e] = fmaf(w, w != 0.f ? f[x][e] : 0.f, o[x][e]);
    }
#pragma unroll
    for (int x = 0; x < kItems; ++x)
      if (c0 + x * 128 < a.rankp) store8(sa + i * ld + c0 + x * 128, o[x]);
  }
  copy_wait<0>();
  __syncthreads();
  const int nc = (warp & 3) * 8, half = warp >> 2, steps = a.rankp / 16;
  float acc[4] = {}, odd[4] = {};
#pragma unroll 2
  for (int x = half; x < steps; x += 4) {
    uint32_t fa[4], fb[4];
    ldsm4(fa, smem_addr(sa + (lane & 15) * ld + x * 16 + (lane >> 4) * 8));
    ldsm4(fb, smem_addr(sb + (nc + (lane & 7)) * ld + x * 16 + ((lane >> 3) & 1) * 8));
    mma16816(acc, fa, fb[0], fb[1]);
    if (x + 2 < steps) {
      ldsm4(fa, smem_addr(sa + (lane & 15) * ld + (x + 2) * 16 + (lane >> 4) * 8));
      ldsm4(fb, smem_addr(sb + (nc + (lane & 7)) * ld + (x + 2) * 16 + ((lane >> 3) & 1) * 8));
      mma16816(odd, fa, fb[0], fb[1]);
    }
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) acc[e] += odd[e];
  if (half) {
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(&s_half[(lane >> 2) + r * 8][nc + (lane & 3) * 2]) = make_float2(acc[2 * r], acc[2 * r + 1]);
  }
  __syncthreads();
  if (half || n0 + nc >= a.vp) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const float2 v = *reinterpret_cast<const float2*>(&s_half[(lane >> 2) + r * 8][nc + (lane & 3) * 2]);
    acc[2 * r] += v.x;
    acc[2 * r + 1] += v.y;
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = m0 + (lane >> 2) + r * 8;
    if (row >= rows) continue;
    const float f = a.out_scale * sigmoid_precise(g[r]);
    *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + row * a.ldo + static_cast<long long>(h) * a.vp + n0 + nc +
                                 (lane & 3) * 2) = bf_pack(acc[2 * r] * f, acc[2 * r + 1] * f);
  }
}

int row_tiles(const LatentParams& a, int mt) { return (a.S * a.H + 16 * mt - 1) / (16 * mt); }
int pick_mt(const LatentParams& a) {
  return a.S * a.H > 16 && attend_smem(a.rankp + a.rotp, 2).stages >= 2 ? 2 : 1;
}

// Key ranges per row tile: fewest rounds of blocks, counting about four tiles per block for its start
// and end, and half a tile per range for the sum over them.
int pick_splits(const LatentParams& a) {
  const int mt = pick_mt(a);
  const int sms = current_sm_count() * (attend_smem(a.rankp + a.rotp, mt).total <= kHalfSmem && mt == 1 ? 2 : 1);
  const int len = a.pos_dev ? a.capacity : a.pos0 + a.S, tiles = (len + kKeys - 1) / kKeys;
  const long long blocks = static_cast<long long>(a.B) * row_tiles(a, mt);
  int best = 1;
  long long cost = -1;
  for (int s = 1; s <= kMaxSplits && s <= tiles; ++s) {
    const long long c = (blocks * s + sms - 1) / sms * ((tiles + s - 1) / s + 4) * 2 + s;
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
  cudaError_t e = allow_smem<latent_attend_kernel<MT, PP>>(bytes);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_attend_kernel<MT, PP>, dim3(p.splits, row_tiles(p.a, MT), p.a.B), dim3(kWarps * 32), bytes, st, p,
                       device_status_word());
}

}  // namespace

bool latent_decode_supported(const LatentParams& a) {
  return a.rankp <= 512 && a.dimp <= 512 && attend_smem(a.rankp + a.rotp, 1).stages >= 2 && a.H <= 65535 &&
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
  const int absorb = 2 * 64 * (a.dimp + 8) * 2, finish = (16 + kValueCols) * (a.rankp + 8) * 2;
  cudaError_t e = allow_smem<latent_absorb_kernel>(absorb);
  if (e != cudaSuccess) return e;
  e = allow_smem<latent_finish_kernel>(finish);
  if (e != cudaSuccess) return e;
  e = launch_kernel(latent_absorb_kernel, dim3((a.rankp + 63) / 64, a.H, (tokens + 63) / 64), dim3(kThreads), absorb, st, p);
  if (e != cudaSuccess) return e;
  const int mt = pick_mt(a);
  if (mt == 1)
    e = a.rankp <= 128 ? launch_attend<1, 1>(p, st) : a.rankp <= 256 ? launch_attend<1, 2>(p, st) : launch_attend<1, 4>(p, st);
  else
    e = a.rankp <= 128 ? launch_attend<2, 1>(p, st) : a.rankp <= 256 ? launch_attend<2, 2>(p, st) : launch_attend<2, 4>(p, st);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_finish_kernel, dim3((a.vp + kValueCols - 1) / kValueCols, a.H, (tokens + 15) / 16), dim3(kThreads), finish, st, p);
}

}  // namespace cdeep

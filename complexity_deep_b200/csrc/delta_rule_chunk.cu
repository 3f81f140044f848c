// The delta rule over a prompt (or a portion of one) in bf16, in chunks of 64 tokens on the tensor cores.
// With B_t = sum of the log decays of a chunk up to and including t, L = B at the chunk's end (both per key
// channel), S the state before the chunk and u_t = beta_t (v_t - (decayed state)^T k_t):
//
//   M_ts = sum_c k_tc k_sc exp(B_tc - B_sc)  (s < t),   A_ts the same with q_t and s <= t
//   u_t + beta_t sum_{s < t} M_ts u_s = beta_t (v_t - S^T (k_t exp(B_t)))
//
// so with T = (I + diag(beta) M)^-1 diag(beta):
//
//   U  = T V - (T K~) S,  K~ = k exp(B)             T, U0 = T V and W = T K~ do not depend on S:
//   O  = Q~ S + A U,      Q~ = q exp(B)             delta_chunk_local_kernel, all chunks in parallel
//   S' = diag(exp L) S + K^ ^T U,  K^ = k exp(L - B)    delta_chunk_scan_kernel, chunk after chunk,
//                                                   a block per head and slice of value columns
//
// M and A are built from 16 x 16 blocks.  Below the diagonal the reference R = B just before the block's
// first row splits exp(B_t - B_s) into two factors of at most one.  On the diagonal R lies in the middle of
// the block, both factors stay finite while the block's decay is below exp(-80) in no channel; a block that
// decays faster takes the differences one by one.
//
// Operands that carry decays, U and the state enter the products as two bf16 parts (16 significant bits);
// sums, decays, T and the state are fp32.
#include "delta_rule.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace cdeep {

namespace {

constexpr int kC = 64;                 // tokens per chunk
constexpr int kThreads = 256;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kMaxSpan = 80.f * kLog2e;
constexpr int kLdM = kC + 4;           // fp32 rows of M and T
constexpr int kLdA = kC + 8;           // bf16 rows of A and of T's parts

struct ChunkParams {
  DeltaParams a;
  int chunks;          // per sequence
  float* u0;           // [B, H, chunks][kC][dvp]
  bf16* w;             // [B, H, chunks][2][kC][dkp] each: high and low parts
  bf16* q;
  bf16* k;
  bf16* att;           // [B, H, chunks][2][kC][kC]
  float* total;        // [B, H, chunks][dkp]: L in the log2 domain
};

__device__ __forceinline__ void store_split2(bf16* hi, bf16* lo, float v0, float v1) {
  uint32_t h, l;
  split_pair(v0, v1, h, l);
  *reinterpret_cast<uint32_t*>(hi) = h;
  *reinterpret_cast<uint32_t*>(lo) = l;
}
__device__ __forceinline__ float2 pair_of(const bf16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf_lo(v), bf_hi(v));
}

// ---------------------------------------------------------------- everything that does not need S
struct LocalSmem {     // byte offsets
  int b, q, k, m, t, tmp, row, total;
};
__host__ __device__ inline LocalSmem local_smem(int dkp, int dvp) {
  LocalSmem s;
  s.b = 0;                                        // [kC][dkp + 4] fp32
  s.q = s.b + kC * (dkp + 4) * 4;                 // [kC][dkp + 8] bf16, later v [kC][dvp + 8]
  s.k = s.q + kC * ((dkp > dvp ? dkp : dvp) + 8) * 2;
  s.m = s.k + kC * (dkp + 8) * 2;                 // [kC][kLdM] fp32, later T's parts [2][kC][kLdA] bf16
  s.t = s.m + 2 * kC * kLdA * 2;                  // [kC][kLdM] fp32
  s.tmp = s.t + kC * kLdM * 4;                    // [3][16][17] fp32 / segment sums [kThreads]
  s.row = s.tmp + 3 * 16 * 17 * 4;                // 1 / |q|, 1 / |k|, beta: [3][kC]
  s.total = s.row + 3 * kC * 4;
  return s;
}

// Adds a 16 x 16 block (t0, s0) of k k^T and q k^T with decays, fast form; `mid`: row of B that serves as
// the reference R (-1: R = 0)
__device__ __forceinline__ void block_products(const float* sB, int ldb, const bf16* sq, const bf16* sk, int ldk,
                                               int dkp, int t0, int s0, int mid, float (&m)[2][4], float (&a)[2][4]) {
  const int lane = threadIdx.x & 31, r = lane >> 2, c0 = (lane & 3) * 2;
  for (int d = 0; d < dkp; d += 16) {
    uint32_t kh[4], kl[4], qh[4], ql[4];
    float2 ref[2];
#pragma unroll
    for (int x = 0; x < 2; ++x)
      ref[x] = mid >= 0 ? *reinterpret_cast<const float2*>(sB + mid * ldb + d + c0 + x * 8) : make_float2(0.f, 0.f);
#pragma unroll
    for (int x = 0; x < 2; ++x)          // columns c0, c0 + 8
#pragma unroll
      for (int y = 0; y < 2; ++y) {      // rows r, r + 8
        const int row = t0 + r + y * 8, col = d + c0 + x * 8;
        const float2 b = *reinterpret_cast<const float2*>(sB + row * ldb + col);
        const float e0 = exp2_approx(b.x - ref[x].x), e1 = exp2_approx(b.y - ref[x].y);
        const float2 kv = pair_of(sk + row * ldk + col), qv = pair_of(sq + row * ldk + col);
        split_pair(kv.x * e0, kv.y * e1, kh[2 * x + y], kl[2 * x + y]);
        split_pair(qv.x * e0, qv.y * e1, qh[2 * x + y], ql[2 * x + y]);
      }
#pragma unroll
    for (int n = 0; n < 2; ++n) {        // keys s0 + 8 n ...
      uint32_t bh[2], bl[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int row = s0 + n * 8 + r, col = d + c0 + x * 8;
        const float2 b = *reinterpret_cast<const float2*>(sB + row * ldb + col);
        const float2 kv = pair_of(sk + row * ldk + col);
        split_pair(kv.x * exp2_approx(ref[x].x - b.x), kv.y * exp2_approx(ref[x].y - b.y), bh[x], bl[x]);
      }
      mma16816(m[n], kh, bl[0], bl[1]);
      mma16816(m[n], kl, bh[0], bh[1]);
      mma16816(m[n], kh, bh[0], bh[1]);
      mma16816(a[n], qh, bl[0], bl[1]);
      mma16816(a[n], ql, bh[0], bh[1]);
      mma16816(a[n], qh, bh[0], bh[1]);
    }
  }
}

__global__ void __launch_bounds__(kThreads, 2)
delta_chunk_local_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const DeltaParams& a = p.a;
  const int n_chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (a.H / a.G);
  const int n = min(kC, a.S - n_chunk * kC);
  const int dkp = a.dkp, dvp = a.dvp, ldb = dkp + 4, ldk = dkp + 8, ldv = dvp + 8, C = delta_channels(a);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const LocalSmem off = local_smem(dkp, dvp);
  float* sB = reinterpret_cast<float*>(smem + off.b);
  bf16* sq = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sk = reinterpret_cast<bf16*>(smem + off.k);
  bf16* sv = sq;                       // once q has been used
  float* sM = reinterpret_cast<float*>(smem + off.m);
  bf16* sTh = reinterpret_cast<bf16*>(smem + off.m);
  bf16* sTl = sTh + kC * kLdA;
  float* sT = reinterpret_cast<float*>(smem + off.t);
  float* s_tmp = reinterpret_cast<float*>(smem + off.tmp);
  float* s_iq = reinterpret_cast<float*>(smem + off.row);
  float* s_ik = s_iq + kC;
  float* s_beta = s_ik + kC;
  const long long row0 = static_cast<long long>(b) * a.S + n_chunk * kC;
  const long long slot = (static_cast<long long>(b) * a.H + h) * p.chunks + n_chunk;

  // ---- rows of q, k, v (zero beyond the sequence), norms, beta
  const bf16* act = static_cast<const bf16*>(a.act) + row0 * C;
  auto copy_rows = [&](bf16* dst, int ld, int col, int width) {       // half a warp per row
    for (int c = (tid & 15) * 8; c < width; c += 128) {
      const bf16* src = act + static_cast<long long>(tid >> 4) * C + col + c;
#pragma unroll
      for (int x = 0; x < kC / (kThreads / 16); ++x, src += static_cast<long long>(kThreads / 16) * C) {
        const int t = (tid >> 4) + x * (kThreads / 16);
        if (t < n) copy16_async(dst + t * ld + c, src);
        else *reinterpret_cast<uint4*>(dst + t * ld + c) = make_uint4(0, 0, 0, 0);
      }
    }
  };
  copy_rows(sq, ldk, g * dkp, dkp);
  copy_rows(sk, ldk, (a.G + g) * dkp, dkp);
  copy_commit();
  if (tid < kC) {
    const bool ok = tid < n;
    s_iq[tid] = ok ? a.inv[(row0 + tid) * 2 * a.G + g] : 0.f;
    s_ik[tid] = ok ? a.inv[(row0 + tid) * 2 * a.G + a.G + g] : 0.f;
    s_beta[tid] = ok ? sigmoid_precise(to_f32(static_cast<const bf16*>(a.b)[(row0 + tid) * a.ldp + h])) : 0.f;
  }
  // ---- B: a thread sums one channel over one segment of the tokens, then adds the segments before it
  {
    int segs = 8;
    while (segs * dkp > kThreads) segs >>= 1;
    const int seg = tid / dkp, c = tid - seg * dkp, len = kC / segs;
    const float rate = a.rate[h] * kLog2e;
    float sum = 0.f;
    if (seg < segs) {
      const float bias = a.dt_bias[h * dkp + c];
      const float* z = a.zg + row0 * a.ldz + h * dkp + c;
      constexpr int kAhead = 8;
      float zv[kAhead], nx[kAhead];
      auto load = [&](int t0, float (&v)[kAhead]) {
#pragma unroll
        for (int x = 0; x < kAhead; ++x) v[x] = t0 + x < n ? z[(t0 + x) * a.ldz] : 0.f;
      };
      const int t_end = (seg + 1) * len;
      load(seg * len, zv);
      for (int t0 = seg * len; t0 < t_end; t0 += kAhead) {
        if (t0 + kAhead < t_end) load(t0 + kAhead, nx);
#pragma unroll
        for (int x = 0; x < kAhead; ++x) {
          if (t0 + x < n) sum -= rate * softplus_fast(zv[x] + bias);
          sB[(t0 + x) * ldb + c] = sum;
          zv[x] = nx[x];
        }
      }
      s_tmp[seg * dkp + c] = sum;
    }
    __syncthreads();
    if (seg < segs) {
      float before = 0.f;
      for (int s = 0; s < seg; ++s) before += s_tmp[s * dkp + c];
      if (seg > 0)
        for (int t = seg * len; t < (seg + 1) * len; ++t) sB[t * ldb + c] += before;
      if (seg == segs - 1) p.total[slot * dkp + c] = before + sum;
    }
  }
  copy_wait<0>();
  __syncthreads();

  // ---- M (scaled by beta) and A, a 16 x 16 block at a time
  {
    bf16* ah = p.att + slot * 2 * kC * kC;
    bf16* al = ah + kC * kC;
    for (int item = warp; item < 10; item += kThreads / 32) {
      // diagonal blocks first, then distances 1, 2, 3
      const int dist = item < 4 ? 0 : item < 7 ? 1 : item < 9 ? 2 : 3;
      const int j = item - (dist == 0 ? 0 : dist == 1 ? 4 : dist == 2 ? 7 : 9), i = j + dist;
      const int t0 = i * 16, s0 = j * 16;
      float m[2][4] = {}, q[2][4] = {};
      bool fast = true;
      if (dist == 0) {
        for (int c = lane; c < dkp; c += 32) fast = fast && sB[t0 * ldb + c] - sB[(t0 + 15) * ldb + c] < kMaxSpan;
        fast = __all_sync(0xffffffffu, fast);
      }
      if (fast) {
        block_products(sB, ldb, sq, sk, ldk, dkp, t0, s0, dist == 0 ? t0 + 7 : t0 - 1, m, q);
      } else {
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int t = t0 + (lane >> 2) + (e >> 1) * 8, s = s0 + y * 8 + (lane & 3) * 2 + (e & 1);
            if (s <= t)
              for (int c = 0; c < dkp; ++c) {
                const float f = exp2_approx(sB[t * ldb + c] - sB[s * ldb + c]) * to_f32(sk[s * ldk + c]);
                m[y][e] = fmaf(to_f32(sk[t * ldk + c]), f, m[y][e]);
                q[y][e] = fmaf(to_f32(sq[t * ldk + c]), f, q[y][e]);
              }
          }
      }
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = t0 + (lane >> 2) + r * 8, s = s0 + y * 8 + (lane & 3) * 2;
          const float ik0 = s_ik[s], ik1 = s_ik[s + 1], f = s_beta[t] * s_ik[t], iq = s_iq[t];
          sM[t * kLdM + s] = s < t ? m[y][2 * r] * f * ik0 : 0.f;
          sM[t * kLdM + s + 1] = s + 1 < t ? m[y][2 * r + 1] * f * ik1 : 0.f;
          store_split2(ah + t * kC + s, al + t * kC + s, s <= t ? q[y][2 * r] * iq * ik0 : 0.f,
                       s + 1 <= t ? q[y][2 * r + 1] * iq * ik1 : 0.f);
        }
    }
  }
  // ---- Q~ and K^
  {
    bf16* qh = p.q + slot * 2 * kC * dkp;
    bf16* kh = p.k + slot * 2 * kC * dkp;
    for (int c = lane * 2; c < dkp; c += 64) {
      const float2 bl = *reinterpret_cast<const float2*>(sB + (kC - 1) * ldb + c);
#pragma unroll 4
      for (int t = warp; t < kC; t += kThreads / 32) {
        const float2 bt = *reinterpret_cast<const float2*>(sB + t * ldb + c);
        const float2 qv = pair_of(sq + t * ldk + c), kv = pair_of(sk + t * ldk + c);
        const float iq = s_iq[t], ik = s_ik[t];
        const int at = t * dkp + c;
        store_split2(qh + at, qh + kC * dkp + at, qv.x * iq * exp2_approx(bt.x), qv.y * iq * exp2_approx(bt.y));
        store_split2(kh + at, kh + kC * dkp + at, kv.x * ik * exp2_approx(bl.x - bt.x), kv.y * ik * exp2_approx(bl.y - bt.y));
      }
    }
  }
  __syncthreads();
  copy_rows(sv, ldv, 2 * a.G * dkp + h * dvp, dvp);
  copy_commit();
  // ---- T = (I + sM)^-1: diagonal blocks by forward substitution, a column per lane ...
  if (warp < 4) {
    const int d0 = warp * 16;
    if (lane < 16) {
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float v = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int s = 0; s < i; ++s) v = fmaf(-sM[(d0 + i) * kLdM + d0 + s], x[s], v);
        x[i] = v;
        sT[(d0 + i) * kLdM + d0 + lane] = v;
      }
    }
  }
  __syncthreads();
  // ... the others by distance: T_ij = -T_ii sum_k M_ik T_kj
  const int br = tid >> 4, bc = tid & 15;
  for (int dist = 1; dist < 4; ++dist) {
    for (int j = 0; j + dist < 4; ++j) {
      const int i = j + dist;
      float v = 0.f;
#pragma unroll 16
      for (int s = j * 16; s < i * 16; ++s) v = fmaf(sM[(i * 16 + br) * kLdM + s], sT[s * kLdM + j * 16 + bc], v);
      s_tmp[(j * 16 + br) * 17 + bc] = v;
    }
    __syncthreads();
    for (int j = 0; j + dist < 4; ++j) {
      const int i = j + dist;
      float v = 0.f;
#pragma unroll
      for (int s = 0; s < 16; ++s) v = fmaf(sT[(i * 16 + br) * kLdM + i * 16 + s], s_tmp[(j * 16 + s) * 17 + bc], v);
      sT[(i * 16 + br) * kLdM + j * 16 + bc] = -v;
    }
    __syncthreads();
  }
  // ---- T diag(beta) in two parts (upper blocks are never read)
  for (int i = tid; i < kC * kC / 2; i += kThreads) {
    const int t = i / (kC / 2), s = (i - t * (kC / 2)) * 2;
    const bool ok = s / 16 <= t / 16;
    const float v0 = ok ? sT[t * kLdM + s] * s_beta[s] : 0.f, v1 = ok ? sT[t * kLdM + s + 1] * s_beta[s + 1] : 0.f;
    store_split2(sTh + t * kLdA + s, sTl + t * kLdA + s, s <= t ? v0 : 0.f, s + 1 <= t ? v1 : 0.f);
  }
  copy_wait<0>();
  __syncthreads();
  // ---- W = T K~ and U0 = T V: a warp takes 16 columns for all 64 rows
  float* u0 = p.u0 + slot * kC * dvp;
  bf16* wh = p.w + slot * 2 * kC * dkp;
  const int k_cols = dkp / 16, v_cols = dvp / 16, r_lo = lane >> 2, c_lo = (lane & 3) * 2;
  for (int item = warp; item < k_cols + v_cols; item += kThreads / 32) {
    const bool is_v = item >= k_cols;
    const int col = (is_v ? item - k_cols : item) * 16;
    float acc[4][2][4] = {};
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t bh[4], bl[4];
      if (is_v) {
        ldsm4_t(bh, smem_addr(sv + (kk * 16 + (lane & 15)) * ldv + col + (lane >> 4) * 8));
      } else {
        // rows kk * 16 + c_lo + {0, 1, 8, 9}, columns col + r_lo and col + 8 + r_lo
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int s = kk * 16 + c_lo + x * 8, c = col + y * 8 + r_lo;
            split_pair(to_f32(sk[s * ldk + c]) * s_ik[s] * exp2_approx(sB[s * ldb + c]),
                       to_f32(sk[(s + 1) * ldk + c]) * s_ik[s + 1] * exp2_approx(sB[(s + 1) * ldb + c]), bh[2 * y + x],
                       bl[2 * y + x]);
          }
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        if (mt < kk) continue;
        uint32_t th[4], tl[4];
        const int at = (mt * 16 + (lane & 15)) * kLdA + kk * 16 + (lane >> 4) * 8;
        ldsm4(th, smem_addr(sTh + at));
        ldsm4(tl, smem_addr(sTl + at));
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          if (!is_v) mma16816(acc[mt][y], th, bl[2 * y], bl[2 * y + 1]);
          mma16816(acc[mt][y], tl, bh[2 * y], bh[2 * y + 1]);
          mma16816(acc[mt][y], th, bh[2 * y], bh[2 * y + 1]);
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < 4; ++mt)
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = mt * 16 + r_lo + r * 8, c = col + y * 8 + c_lo;
          if (is_v)
            *reinterpret_cast<float2*>(u0 + t * dvp + c) = make_float2(acc[mt][y][2 * r], acc[mt][y][2 * r + 1]);
          else
            store_split2(wh + t * dkp + c, wh + (kC + t) * dkp + c, acc[mt][y][2 * r], acc[mt][y][2 * r + 1]);
        }
  }
}

// ---------------------------------------------------------------- chunk after chunk
struct ScanSmem {      // byte offsets
  int w, q, k, att, u, s, total;
};
__host__ __device__ inline ScanSmem scan_smem(int dkp, int nb) {
  ScanSmem s;
  s.w = 0;                                        // [2][kC][dkp + 8] bf16 each
  s.q = s.w + 2 * kC * (dkp + 8) * 2;
  s.k = s.q + 2 * kC * (dkp + 8) * 2;
  s.att = s.k + 2 * kC * (dkp + 8) * 2;           // [2][kC][kLdA]
  s.u = s.att + 2 * kC * kLdA * 2;                // [2][kC][nb + 8]
  s.s = s.u + 2 * kC * (nb + 8) * 2;              // [2][dkp][nb + 8]
  s.total = s.s + 2 * dkp * (nb + 8) * 2;
  return s;
}

// NB value columns per block; the NW warps tile the state as KT row tiles of 16 (dkp <= 16 KT) by NW / KT
// column slices, and the chunk's rows as four row tiles by NW / 4 column slices
template <int NB, int KT, int NW>
__global__ void __launch_bounds__(NW * 32, 1)
delta_chunk_scan_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const DeltaParams& a = p.a;
  constexpr int kThreads = NW * 32;
  constexpr int kSlices = NW / KT, kSN = NB / 8 / kSlices;    // n-tiles of the state per warp
  constexpr int kON = NB / 8 / (NW / 4);                      // n-tiles of U and O per warp
  static_assert(kSN % 2 == 0 && kON % 2 == 0, "column slices are pairs of n-tiles");
  constexpr int ldn = NB + 8;
  const int col0 = blockIdx.x * NB, h = blockIdx.y, b = blockIdx.z;
  const int dkp = a.dkp, dvp = a.dvp, ldk = dkp + 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r_lo = lane >> 2, c_lo = (lane & 3) * 2;
  const ScanSmem off = scan_smem(dkp, NB);
  bf16* sw = reinterpret_cast<bf16*>(smem + off.w);
  bf16* sq = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sk = reinterpret_cast<bf16*>(smem + off.k);
  bf16* sa = reinterpret_cast<bf16*>(smem + off.att);
  bf16* su = reinterpret_cast<bf16*>(smem + off.u);
  bf16* sS = reinterpret_cast<bf16*>(smem + off.s);
  const long long slot0 = (static_cast<long long>(b) * a.H + h) * p.chunks;
  const long long row0 = static_cast<long long>(b) * a.S;

  auto fetch = [&](bf16* dst, const bf16* src) {              // [2][kC][dkp] -> [2][kC][ldk], half a warp per row
    const int c = (tid & 15) * 8;                             // dkp <= 128
    if (c >= dkp) return;
#pragma unroll
    for (int x = 0; x < 2 * kC / (kThreads / 16); ++x) {
      const int t = (tid >> 4) + x * (kThreads / 16);
      copy16_async(dst + t * ldk + c, src + t * dkp + c);
    }
  };
  auto fetch_w = [&](int n) { fetch(sw, p.w + (slot0 + n) * 2 * kC * dkp); };
  auto fetch_rest = [&](int n) {
    fetch(sq, p.q + (slot0 + n) * 2 * kC * dkp);
    fetch(sk, p.k + (slot0 + n) * 2 * kC * dkp);
    const bf16* src = p.att + (slot0 + n) * 2 * kC * kC;
#pragma unroll
    for (int x = 0; x < 2 * kC * kC / 8 / kThreads; ++x) {
      const int i = tid + x * kThreads, t = i / (kC / 8), c = (i - t * (kC / 8)) * 8;
      copy16_async(sa + t * kLdA + c, src + t * kC + c);
    }
  };
  fetch_w(0);
  copy_commit();
  fetch_rest(0);
  copy_commit();

  // this warp's part of the state
  const int st = warp % KT, sc = (warp / KT) * (kSN * 8);
  const bool st_ok = st * 16 < dkp;
  float S[kSN][4];
  float* state = a.state + (static_cast<long long>(b) * a.H + h) * dkp * dvp + col0;
#pragma unroll
  for (int x = 0; x < kSN; ++x)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = st * 16 + r_lo + r * 8, c = sc + x * 8 + c_lo;
      const float2 v = (st_ok && col0 + c < dvp) ? *reinterpret_cast<const float2*>(state + static_cast<long long>(row) * dvp + c)
                                                 : make_float2(0.f, 0.f);
      S[x][2 * r] = v.x;
      S[x][2 * r + 1] = v.y;
    }
  auto put_state = [&]() {
    if (!st_ok) return;
#pragma unroll
    for (int x = 0; x < kSN; ++x)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int at = (st * 16 + r_lo + r * 8) * ldn + sc + x * 8 + c_lo;
        store_split2(sS + at, sS + dkp * ldn + at, S[x][2 * r], S[x][2 * r + 1]);
      }
  };
  put_state();

  const int mt = warp & 3, oc = (warp >> 2) * (kON * 8);       // this warp's rows and columns of U and O
  // acc += x S for this warp's tile; x: [2][kC][ldk] in shared memory
  auto times_state = [&](const bf16* x, float (&acc)[kON][4]) {
#pragma unroll 2
    for (int d = 0; d < dkp; d += 16) {
      uint32_t ah[4], al[4];
      const int at = (mt * 16 + (lane & 15)) * ldk + d + (lane >> 4) * 8;
      ldsm4(ah, smem_addr(x + at));
      ldsm4(al, smem_addr(x + kC * ldk + at));
#pragma unroll
      for (int y = 0; y < kON / 2; ++y) {
        uint32_t bh[4], bl[4];
        const int bt = (d + (lane & 15)) * ldn + oc + y * 16 + (lane >> 4) * 8;
        ldsm4_t(bh, smem_addr(sS + bt));
        ldsm4_t(bl, smem_addr(sS + dkp * ldn + bt));
#pragma unroll
        for (int z = 0; z < 2; ++z) {
          mma16816(acc[2 * y + z], ah, bl[2 * z], bl[2 * z + 1]);
          mma16816(acc[2 * y + z], al, bh[2 * z], bh[2 * z + 1]);
          mma16816(acc[2 * y + z], ah, bh[2 * z], bh[2 * z + 1]);
        }
      }
    }
  };

  for (int n = 0; n < p.chunks; ++n) {
    const long long slot = slot0 + n;
    // U0 and the decays of this chunk, in flight during the first product
    float2 u0[kON][2];
#pragma unroll
    for (int x = 0; x < kON; ++x)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = mt * 16 + r_lo + r * 8, c = col0 + oc + x * 8 + c_lo;
        u0[x][r] = c < dvp ? *reinterpret_cast<const float2*>(p.u0 + (slot * kC + t) * dvp + c) : make_float2(0.f, 0.f);
      }
    float decay[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) decay[r] = st_ok ? p.total[slot * dkp + st * 16 + r_lo + r * 8] : 0.f;
    copy_wait<1>();
    __syncthreads();                   // W of this chunk and the state are in place
    {
      float acc[kON][4] = {};
      times_state(sw, acc);
#pragma unroll
      for (int x = 0; x < kON; ++x)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int at = (mt * 16 + r_lo + r * 8) * ldn + oc + x * 8 + c_lo;
          store_split2(su + at, su + kC * ldn + at, u0[x][r].x - acc[x][2 * r], u0[x][r].y - acc[x][2 * r + 1]);
        }
    }
    copy_wait<0>();
    __syncthreads();                   // U, Q~, K^ and A are in place, W is free
    if (n + 1 < p.chunks) fetch_w(n + 1);
    copy_commit();
    {
      float acc[kON][4] = {};
      times_state(sq, acc);
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk > mt) break;
        uint32_t ah[4], al[4];
        const int at = (mt * 16 + (lane & 15)) * kLdA + kk * 16 + (lane >> 4) * 8;
        ldsm4(ah, smem_addr(sa + at));
        ldsm4(al, smem_addr(sa + kC * kLdA + at));
#pragma unroll
        for (int y = 0; y < kON / 2; ++y) {
          uint32_t bh[4], bl[4];
          const int bt = (kk * 16 + (lane & 15)) * ldn + oc + y * 16 + (lane >> 4) * 8;
          ldsm4_t(bh, smem_addr(su + bt));
          ldsm4_t(bl, smem_addr(su + kC * ldn + bt));
#pragma unroll
          for (int z = 0; z < 2; ++z) {
            mma16816(acc[2 * y + z], ah, bl[2 * z], bl[2 * z + 1]);
            mma16816(acc[2 * y + z], al, bh[2 * z], bh[2 * z + 1]);
            mma16816(acc[2 * y + z], ah, bh[2 * z], bh[2 * z + 1]);
          }
        }
      }
#pragma unroll
      for (int x = 0; x < kON; ++x)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = n * kC + mt * 16 + r_lo + r * 8, c = col0 + oc + x * 8 + c_lo;
          if (t < a.S && c < dvp)
            *reinterpret_cast<float2*>(a.o_raw + (row0 + t) * (a.H * dvp) + static_cast<long long>(h) * dvp + c) =
                make_float2(acc[x][2 * r], acc[x][2 * r + 1]);
        }
    }
    if (st_ok) {
#pragma unroll
      for (int x = 0; x < kSN; ++x) {
        const float f0 = exp2_approx(decay[0]), f1 = exp2_approx(decay[1]);
        S[x][0] *= f0;
        S[x][1] *= f0;
        S[x][2] *= f1;
        S[x][3] *= f1;
      }
#pragma unroll
      for (int kk = 0; kk < kC / 16; ++kk) {
        uint32_t ah[4], al[4];
        const int at = (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + st * 16 + ((lane >> 3) & 1) * 8;
        ldsm4_t(ah, smem_addr(sk + at));
        ldsm4_t(al, smem_addr(sk + kC * ldk + at));
#pragma unroll
        for (int y = 0; y < kSN / 2; ++y) {
          uint32_t bh[4], bl[4];
          const int bt = (kk * 16 + (lane & 15)) * ldn + sc + y * 16 + (lane >> 4) * 8;
          ldsm4_t(bh, smem_addr(su + bt));
          ldsm4_t(bl, smem_addr(su + kC * ldn + bt));
#pragma unroll
          for (int z = 0; z < 2; ++z) {
            mma16816(S[2 * y + z], ah, bl[2 * z], bl[2 * z + 1]);
            mma16816(S[2 * y + z], al, bh[2 * z], bh[2 * z + 1]);
            mma16816(S[2 * y + z], ah, bh[2 * z], bh[2 * z + 1]);
          }
        }
      }
    }
    __syncthreads();                   // nobody reads the state, Q~, K^, A or U any more
    if (n + 1 < p.chunks) fetch_rest(n + 1);
    copy_commit();
    put_state();
  }
  if (!st_ok) return;
#pragma unroll
  for (int x = 0; x < kSN; ++x)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = st * 16 + r_lo + r * 8, c = sc + x * 8 + c_lo;
      if (col0 + c < dvp)
        *reinterpret_cast<float2*>(state + static_cast<long long>(row) * dvp + c) = make_float2(S[x][2 * r], S[x][2 * r + 1]);
    }
}

int chunk_count(int S) { return (S + kC - 1) / kC; }

template <int NB, int KT, int NW>
cudaError_t launch_scan(const ChunkParams& p, cudaStream_t st) {
  const int bytes = scan_smem(p.a.dkp, NB).total;
  cudaError_t e = allow_smem<delta_chunk_scan_kernel<NB, KT, NW>>(bytes);
  if (e != cudaSuccess) return e;
  return launch_kernel(delta_chunk_scan_kernel<NB, KT, NW>, dim3((p.a.dvp + NB - 1) / NB, p.a.H, p.a.B), dim3(NW * 32),
                       bytes, st, p);
}

// Columns per block: rounds of blocks (one block per SM) times the measured relative time of a block
int pick_columns(const DeltaParams& a) {
  const int sms = current_sm_count();
  auto cost = [&](int nb, int t) {
    const long long blocks = static_cast<long long>(a.B) * a.H * ((a.dvp + nb - 1) / nb);
    return (blocks + sms - 1) / sms * t;
  };
  const long long c32 = cost(32, 75), c64 = cost(64, 100), c128 = cost(128, 130);
  if (c128 < c64 && c128 < c32) return 128;
  return c64 <= c32 ? 64 : 32;
}

struct Sizes {         // bytes per (sequence, head, chunk)
  size_t u0, wide, att, total;
};
Sizes sizes(const DeltaParams& a) {
  return {static_cast<size_t>(kC) * a.dvp * 4, static_cast<size_t>(2) * kC * a.dkp * 2, static_cast<size_t>(2) * kC * kC * 2,
          static_cast<size_t>(a.dkp) * 4};
}

}  // namespace

bool delta_chunk_supported(const DeltaParams& a) {
  return a.dkp <= 128 && a.dvp <= 256 && local_smem(a.dkp, a.dvp).total <= 227 * 1024 && a.H <= 65535;
}

size_t delta_chunk_workspace_bytes(const DeltaParams& a) {
  const Sizes s = sizes(a);
  return static_cast<size_t>(a.B) * a.H * chunk_count(a.S) * (s.u0 + 3 * s.wide + s.att + s.total);
}

cudaError_t launch_delta_chunk(const DeltaParams& a, void* ws, cudaStream_t st) {
  if (a.B == 0 || a.S == 0) return cudaSuccess;
  ChunkParams p;
  p.a = a;
  p.chunks = chunk_count(a.S);
  const Sizes s = sizes(a);
  const size_t slots = static_cast<size_t>(a.B) * a.H * p.chunks;
  char* at = static_cast<char*>(ws);
  auto take = [&](size_t bytes) {
    char* r = at;
    at += slots * bytes;
    return r;
  };
  p.u0 = reinterpret_cast<float*>(take(s.u0));
  p.w = reinterpret_cast<bf16*>(take(s.wide));
  p.q = reinterpret_cast<bf16*>(take(s.wide));
  p.k = reinterpret_cast<bf16*>(take(s.wide));
  p.att = reinterpret_cast<bf16*>(take(s.att));
  p.total = reinterpret_cast<float*>(take(s.total));
  const int bytes = local_smem(a.dkp, a.dvp).total;
  cudaError_t e = allow_smem<delta_chunk_local_kernel>(bytes);
  if (e != cudaSuccess) return e;
  e = launch_kernel(delta_chunk_local_kernel, dim3(p.chunks, a.H, a.B), dim3(kThreads), bytes, st, p);
  if (e != cudaSuccess) return e;
  const int nb = pick_columns(a);
  if (a.dkp <= 32) return launch_scan<64, 2, 8>(p, st);
  if (a.dkp <= 64)
    return nb == 32 ? launch_scan<32, 4, 8>(p, st) : nb == 64 ? launch_scan<64, 4, 8>(p, st) : launch_scan<128, 4, 16>(p, st);
  return nb == 32 ? launch_scan<32, 8, 8>(p, st) : nb == 64 ? launch_scan<64, 8, 8>(p, st) : launch_scan<128, 8, 16>(p, st);
}

}  // namespace cdeep

// Gated linear attention of a prompt (or a portion of one) in bf16, in chunks of 64 tokens on the
// tensor cores.  With B_t = sum of the log decays of a chunk up to and including t, and L = B at the
// chunk's end, all per key channel:
//
//   U    = sum_s (k_s exp(L - B_s)) v_s^T                          gla_chunk_update_kernel
//   S'   = diag(exp(L)) S + U,  S before every chunk kept          gla_chunk_scan_kernel
//   o_t  = S^T (q_t exp(B_t)) + sum_{s <= t} A_ts v_s,             gla_chunk_output_kernel
//   A_ts = sum_c q_tc k_sc exp(B_tc - B_sc)                        (+ head norm and gate)
//
// A_ts is a product of q_t exp(B_t - R) and k_s exp(R - B_s) for any reference R per channel.  With
// R = L / 2 both factors stay within exp(+-|L| / 2), so as long as |L| < 120 for every channel of
// the head nothing leaves the fp32 (= bf16) exponent range; R then also moves into S's rows, as
// exp(R) S.  A chunk that decays faster takes the differences B_t - B_s one by one instead.
//
// Operands that carry decays, and the state, enter the products as two bf16 parts (16 significant
// bits); v is bf16 as projected; sums, decays, A and the state are fp32.
#include "kernels.h"
#include "linear_attention.cuh"
#include "mma.cuh"

namespace cdeep {

namespace {

constexpr int kC = 64;                 // tokens per chunk
constexpr int kThreads = 256;
constexpr float kMaxSpan = 120.f;
constexpr int kLdA = kC + 8;
constexpr int kBatch = 8;              // tokens loaded at a time by a channel's thread (divides a segment)

__host__ __device__ inline int segments(int dkp) {   // threads per channel, each with kC / segments tokens
  int s = 8;
  while (s > 1 && s * dkp > kThreads) s >>= 1;
  return s;
}

struct ChunkParams {
  LinearAttnParams a;
  int chunks;            // per sequence
  float* u;              // [B, H, chunks, dkp, dvp]: U, then S before the chunk
  float* total;          // [B, H, chunks, dkp]: L
};

// Sums of a thread's (channel, segment); `start` = sum before the segment, `total` = of the chunk.
// Channels dkp <= 256; one barrier inside.
struct Sums {
  int c, t_lo, t_hi;     // channel (-1: thread idle) and its tokens of the chunk
  float start, total;
};
__device__ __forceinline__ Sums chunk_sums(const LinearAttnParams& a, const float* ld, int n, float* s_seg) {
  const int segs = segments(a.dkp), len = kC / segs, ch = a.H * a.dkp;
  Sums r;
  const int seg = threadIdx.x / a.dkp;
  r.c = seg < segs ? static_cast<int>(threadIdx.x) - seg * a.dkp : -1;
  r.t_lo = seg * len;
  r.t_hi = r.t_lo + len;
  float sum = 0.f;
  if (r.c >= 0) {
    for (int t0 = r.t_lo; t0 < r.t_hi; t0 += kBatch) {
      float v[kBatch];
#pragma unroll
      for (int x = 0; x < kBatch; ++x) v[x] = t0 + x < n ? ld[static_cast<long long>(t0 + x) * ch + r.c] : 0.f;
#pragma unroll
      for (int x = 0; x < kBatch; ++x) sum += v[x];
    }
    s_seg[seg * a.dkp + r.c] = sum;
  }
  __syncthreads();
  r.start = r.total = 0.f;
  if (r.c >= 0)
    for (int s = 0; s < segs; ++s) {
      const float v = s_seg[s * a.dkp + r.c];
      if (s < seg) r.start += v;
      r.total += v;
    }
  return r;
}

__device__ __forceinline__ void store_split(bf16* hi, bf16* lo, int at, float v) {
  const bf16 h = __float2bfloat16_rn(v);
  hi[at] = h;
  lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
}

// rows of v of the chunk, zero beyond n
__device__ __forceinline__ void load_v(const LinearAttnParams& a, long long row0, int h, int n, bf16* sv, int ldv) {
  const bf16* v = static_cast<const bf16*>(a.v) + row0 * a.ldp + static_cast<long long>(h) * a.dvp;
  const int per = a.dvp / 8;
  for (int idx = threadIdx.x; idx < kC * per; idx += kThreads) {
    const int t = idx / per, c = (idx - t * per) * 8;
    if (t < n) copy16_async(sv + t * ldv + c, v + t * a.ldp + c);
    else *reinterpret_cast<uint4*>(sv + t * ldv + c) = make_uint4(0, 0, 0, 0);
  }
  copy_commit();
}

__global__ void __launch_bounds__(kThreads)
gla_chunk_update_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const LinearAttnParams& a = p.a;
  const int n_chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int n = min(kC, a.S - n_chunk * kC);
  const int ldk = a.dkp + 8, ldv = a.dvp + 8, ch = a.H * a.dkp;
  bf16* skh = reinterpret_cast<bf16*>(smem);
  bf16* skl = skh + kC * ldk;
  bf16* sv = skl + kC * ldk;
  float* s_seg = reinterpret_cast<float*>(sv + kC * ldv);
  const long long row0 = static_cast<long long>(b) * a.S + n_chunk * kC;
  load_v(a, row0, h, n, sv, ldv);
  const float* ld = a.log_decay + row0 * ch + h * a.dkp;
  const bf16* k = static_cast<const bf16*>(a.k) + row0 * a.ldp + static_cast<long long>(h) * a.dkp;
  const long long slot = (static_cast<long long>(b) * a.H + h) * p.chunks + n_chunk;
  const Sums s = chunk_sums(a, ld, n, s_seg);
  if (s.c >= 0) {
    float cum = s.start;
    for (int t0 = s.t_lo; t0 < s.t_hi; t0 += kBatch) {
      float d[kBatch];
      bf16 kv[kBatch];
#pragma unroll
      for (int x = 0; x < kBatch; ++x) {
        const bool ok = t0 + x < n;
        d[x] = ok ? ld[static_cast<long long>(t0 + x) * ch + s.c] : 0.f;
        kv[x] = ok ? k[(t0 + x) * a.ldp + s.c] : __float2bfloat16_rn(0.f);
      }
#pragma unroll
      for (int x = 0; x < kBatch; ++x) {
        cum += d[x];
        store_split(skh, skl, (t0 + x) * ldk + s.c, to_f32(kv[x]) * expf(s.total - cum));
      }
    }
    if (s.t_lo == 0) p.total[slot * a.dkp + s.c] = s.total;
  }
  copy_wait<0>();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* u = p.u + slot * a.dkp * a.dvp;
  const int m_tiles = a.dkp / 16, n_blocks = (a.dvp + 63) / 64;
  for (int item = warp; item < m_tiles * n_blocks; item += kThreads / 32) {
    const int mt = item % m_tiles, nb = item / m_tiles;
    float acc[8][4] = {};
#pragma unroll
    for (int kk = 0; kk < kC / 16; ++kk) {
      const int at = (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + mt * 16 + ((lane >> 3) & 1) * 8;
      uint32_t ah[4], al[4];
      ldsm4_t(ah, smem_addr(skh + at));
      ldsm4_t(al, smem_addr(skl + at));
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int col = nb * 64 + x * 16;
        if (col < a.dvp) {
          uint32_t vb[4];
          ldsm4_t(vb, smem_addr(sv + (kk * 16 + (lane & 15)) * ldv + col + (lane >> 4) * 8));
          mma16816(acc[2 * x], al, vb[0], vb[1]);
          mma16816(acc[2 * x + 1], al, vb[2], vb[3]);
          mma16816(acc[2 * x], ah, vb[0], vb[1]);
          mma16816(acc[2 * x + 1], ah, vb[2], vb[3]);
        }
      }
    }
#pragma unroll
    for (int x = 0; x < 8; ++x) {
      const int col = nb * 64 + x * 8 + (lane & 3) * 2;
      if (nb * 64 + x * 8 < a.dvp) {
        float* dst = u + static_cast<long long>(mt * 16 + (lane >> 2)) * a.dvp + col;
        *reinterpret_cast<float2*>(dst) = make_float2(acc[x][0], acc[x][1]);
        *reinterpret_cast<float2*>(dst + 8ll * a.dvp) = make_float2(acc[x][2], acc[x][3]);
      }
    }
  }
}

// S before every chunk (in place of U) and the state after the last one; a thread owns four columns
// of one row of one head's state
__global__ void __launch_bounds__(kThreads)
gla_chunk_scan_kernel(const ChunkParams p) {
  pdl_enter();
  const LinearAttnParams& a = p.a;
  const long long per = static_cast<long long>(a.dkp) * a.dvp / 4;
  const long long idx = blockIdx.x * static_cast<long long>(kThreads) + threadIdx.x;
  if (idx >= per * a.B * a.H) return;
  const long long bh = idx / per, e = idx - bh * per;
  const int c = static_cast<int>(e / (a.dvp / 4));
  float4* st = reinterpret_cast<float4*>(a.state) + bh * per + e;
  float4* u = reinterpret_cast<float4*>(p.u) + bh * p.chunks * per + e;
  const float* tot = p.total + bh * p.chunks * a.dkp + c;
  float4 s = *st;
  constexpr int kAhead = 8;
  for (int n0 = 0; n0 < p.chunks; n0 += kAhead) {
    float4 v[kAhead];
    float d[kAhead];
#pragma unroll
    for (int x = 0; x < kAhead; ++x)
      if (n0 + x < p.chunks) {
        v[x] = u[(n0 + x) * per];
        d[x] = tot[(n0 + x) * a.dkp];
      }
#pragma unroll
    for (int x = 0; x < kAhead; ++x)
      if (n0 + x < p.chunks) {
        u[(n0 + x) * per] = s;
        const float f = expf(d[x]);
        s.x = fmaf(f, s.x, v[x].x);
        s.y = fmaf(f, s.y, v[x].y);
        s.z = fmaf(f, s.z, v[x].z);
        s.w = fmaf(f, s.w, v[x].w);
      }
  }
  *st = s;
}

struct OutSmem {   // byte offsets
  int q, k, v, a, seg, ref, rows, total;
};
__host__ __device__ inline OutSmem out_smem(int dkp, int dvp) {
  OutSmem s;
  s.q = 0;                                        // q parts: [2][kC][dkp + 8] bf16
  s.k = s.q + 2 * kC * (dkp + 8) * 2;             // k parts, or B as fp32 [kC][dkp]
  s.v = s.k + 2 * kC * (dkp + 8) * 2;             // [kC][dvp + 8]
  s.a = s.v + kC * (dvp + 8) * 2;                 // A parts: [2][kC][kLdA]
  s.seg = s.a + 2 * kC * kLdA * 2;                // [8][dkp] at most kThreads
  s.ref = s.seg + kThreads * 4;                   // [dkp]
  s.rows = s.ref + dkp * 4;                       // [8][kC]
  s.total = s.rows + 8 * kC * 4;
  return s;
}

// MT row tiles of 16 tokens per warp (4: eight column slots of 16; 2: four slots, two halves of the
// rows), NJ rounds of column slots
template <int MT, int NJ>
__global__ void __launch_bounds__(kThreads)
gla_chunk_output_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char smem[];
  pdl_enter();
  const LinearAttnParams& a = p.a;
  const int n_chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int n = min(kC, a.S - n_chunk * kC);
  const int dkp = a.dkp, dvp = a.dvp, ldk = dkp + 8, ldv = dvp + 8, ch = a.H * dkp;
  const OutSmem off = out_smem(dkp, dvp);
  bf16* sqh = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sql = sqh + kC * ldk;
  bf16* skh = reinterpret_cast<bf16*>(smem + off.k);
  bf16* skl = skh + kC * ldk;
  float* sB = reinterpret_cast<float*>(smem + off.k);
  bf16* sv = reinterpret_cast<bf16*>(smem + off.v);
  bf16* sah = reinterpret_cast<bf16*>(smem + off.a);
  bf16* sal = sah + kC * kLdA;
  float* s_seg = reinterpret_cast<float*>(smem + off.seg);
  float* s_ref = reinterpret_cast<float*>(smem + off.ref);
  float* s_rows = reinterpret_cast<float*>(smem + off.rows);
  const long long row0 = static_cast<long long>(b) * a.S + n_chunk * kC;
  load_v(a, row0, h, n, sv, ldv);
  const float* ld = a.log_decay + row0 * ch + h * dkp;
  const bf16* q = static_cast<const bf16*>(a.q) + row0 * a.ldp + static_cast<long long>(h) * dkp;
  const bf16* k = static_cast<const bf16*>(a.k) + row0 * a.ldp + static_cast<long long>(h) * dkp;
  const Sums s = chunk_sums(a, ld, n, s_seg);
  const bool fast = !__syncthreads_or(s.c >= 0 && !(-s.total < kMaxSpan));
  const float ref = fast ? 0.5f * s.total : 0.f;
  if (s.c >= 0) {
    float cum = s.start;
    for (int t0 = s.t_lo; t0 < s.t_hi; t0 += kBatch) {
      float d[kBatch];
      bf16 qv[kBatch], kv[kBatch];
#pragma unroll
      for (int x = 0; x < kBatch; ++x) {
        const bool ok = t0 + x < n;
        d[x] = ok ? ld[static_cast<long long>(t0 + x) * ch + s.c] : 0.f;
        qv[x] = ok ? q[(t0 + x) * a.ldp + s.c] : __float2bfloat16_rn(0.f);
        kv[x] = ok ? k[(t0 + x) * a.ldp + s.c] : __float2bfloat16_rn(0.f);
      }
#pragma unroll
      for (int x = 0; x < kBatch; ++x) {
        const int t = t0 + x;
        cum += d[x];
        store_split(sqh, sql, t * ldk + s.c, to_f32(qv[x]) * a.q_scale * expf(cum - ref));
        if (fast) store_split(skh, skl, t * ldk + s.c, to_f32(kv[x]) * expf(ref - cum));
        else sB[t * dkp + s.c] = cum;
      }
    }
    if (s.t_lo == 0) s_ref[s.c] = expf(ref);
  }
  copy_wait<0>();
  __syncthreads();

  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r_lo = lane >> 2, c_lo = (lane & 3) * 2;
  // ---------------------------------------------------------------- A
  if (fast) {
    const int mt = warp >> 1, s0 = (warp & 1) * 32;
    float acc[4][4] = {};
    if (s0 <= mt * 16 + 15) {
      for (int d = 0; d < dkp; d += 16) {
        const int qa = (mt * 16 + (lane & 15)) * ldk + d + (lane >> 4) * 8;
        uint32_t ah[4], al[4];
        ldsm4(ah, smem_addr(sqh + qa));
        ldsm4(al, smem_addr(sql + qa));
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int ka = (s0 + x * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + d + ((lane >> 3) & 1) * 8;
          uint32_t bh[4], bl[4];
          ldsm4(bh, smem_addr(skh + ka));
          ldsm4(bl, smem_addr(skl + ka));
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma16816(acc[2 * x + y], ah, bl[2 * y], bl[2 * y + 1]);
            mma16816(acc[2 * x + y], al, bh[2 * y], bh[2 * y + 1]);
            mma16816(acc[2 * x + y], ah, bh[2 * y], bh[2 * y + 1]);
          }
        }
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = mt * 16 + r_lo + r * 8, sc = s0 + x * 8 + c_lo;
        uint32_t hi, lo;
        split_pair(sc <= t ? acc[x][2 * r] : 0.f, sc + 1 <= t ? acc[x][2 * r + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(sah + t * kLdA + sc) = hi;
        *reinterpret_cast<uint32_t*>(sal + t * kLdA + sc) = lo;
      }
  } else {
    for (int idx = threadIdx.x; idx < kC * kC; idx += kThreads) {
      const int t = idx / kC, sc = idx - t * kC;
      float v = 0.f;
      if (sc <= t && t < n) {
        for (int c = 0; c < dkp; ++c)
          v += to_f32(q[t * a.ldp + c]) * to_f32(k[sc * a.ldp + c]) * expf(sB[t * dkp + c] - sB[sc * dkp + c]);
        v *= a.q_scale;
      }
      store_split(sah, sal, t * kLdA + sc, v);
    }
  }
  __syncthreads();

  // ---------------------------------------------------------------- o = S^T q~ + A v
  constexpr int kSlots = MT == 4 ? 8 : 4;
  const int slot = warp % kSlots, m0 = (warp / kSlots) * MT;     // this warp's column slot and first row tile
  const float* S = p.u + ((static_cast<long long>(b) * a.H + h) * p.chunks + n_chunk) * dkp * dvp;
  float acc[NJ][MT][2][4];
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][m][y][e] = 0.f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int col = (j * kSlots + slot) * 16;
    if (col >= dvp) continue;
    // the state's fragments come straight from memory: rows (lane % 4) * 2 + {0, 1, 8, 9}, column lane / 4
    constexpr int kFetch = NJ == 1 ? 4 : 2;              // steps of 16 rows in flight
    for (int d0 = 0; d0 < dkp; d0 += 16 * kFetch) {
      float f[kFetch][8];
#pragma unroll
      for (int z = 0; z < kFetch; ++z)
        if (d0 + z * 16 < dkp) {
#pragma unroll
          for (int y = 0; y < 2; ++y)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int r = d0 + z * 16 + c_lo + (e & 1) + (e >> 1) * 8;
              f[z][y * 4 + e] = S[static_cast<long long>(r) * dvp + col + y * 8 + r_lo];
            }
        }
#pragma unroll
      for (int z = 0; z < kFetch; ++z) {
        const int d = d0 + z * 16;
        if (d >= dkp) break;
        const float2 fa = *reinterpret_cast<const float2*>(s_ref + d + c_lo);
        const float2 fb = *reinterpret_cast<const float2*>(s_ref + d + c_lo + 8);
        uint32_t bh[4], bl[4];
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          split_pair(f[z][y * 4] * fa.x, f[z][y * 4 + 1] * fa.y, bh[2 * y], bl[2 * y]);
          split_pair(f[z][y * 4 + 2] * fb.x, f[z][y * 4 + 3] * fb.y, bh[2 * y + 1], bl[2 * y + 1]);
        }
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const int qa = ((m0 + m) * 16 + (lane & 15)) * ldk + d + (lane >> 4) * 8;
          uint32_t ah[4], al[4];
          ldsm4(ah, smem_addr(sqh + qa));
          ldsm4(al, smem_addr(sql + qa));
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma16816(acc[j][m][y], ah, bl[2 * y], bl[2 * y + 1]);
            mma16816(acc[j][m][y], al, bh[2 * y], bh[2 * y + 1]);
            mma16816(acc[j][m][y], ah, bh[2 * y], bh[2 * y + 1]);
          }
        }
      }
    }
#pragma unroll
    for (int kk = 0; kk < kC / 16; ++kk) {
      uint32_t vb[4];
      ldsm4_t(vb, smem_addr(sv + (kk * 16 + (lane & 15)) * ldv + col + (lane >> 4) * 8));
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        if (kk > m0 + m) continue;
        const int at = ((m0 + m) * 16 + (lane & 15)) * kLdA + kk * 16 + (lane >> 4) * 8;
        uint32_t ah[4], al[4];
        ldsm4(ah, smem_addr(sah + at));
        ldsm4(al, smem_addr(sal + at));
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          mma16816(acc[j][m][y], al, vb[2 * y], vb[2 * y + 1]);
          mma16816(acc[j][m][y], ah, vb[2 * y], vb[2 * y + 1]);
        }
      }
    }
  }

  // ---------------------------------------------------------------- head norm, gate, store
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int y = 0; y < 2; ++y)
          ss += acc[j][m][y][2 * r] * acc[j][m][y][2 * r] + acc[j][m][y][2 * r + 1] * acc[j][m][y][2 * r + 1];
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if ((lane & 3) == 0) s_rows[slot * kC + (m0 + m) * 16 + r_lo + r * 8] = ss;
    }
  __syncthreads();
  const bf16* gate = static_cast<const bf16*>(a.gate) + row0 * a.ldp + static_cast<long long>(h) * dvp;
  const bf16* w = static_cast<const bf16*>(a.norm_w);
  bf16* out = static_cast<bf16*>(a.out) + row0 * a.ldo + static_cast<long long>(h) * dvp;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = (m0 + m) * 16 + r_lo + r * 8;
      if (t >= n) continue;
      float ss = 0.f;
#pragma unroll
      for (int x = 0; x < kSlots; ++x) ss += s_rows[x * kC + t];
      const float inv = 1.0f / sqrtf(ss / static_cast<float>(a.dv) + a.eps);
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int col = (j * kSlots + slot) * 16 + y * 8 + c_lo;
          if (col >= dvp) continue;
          const uint32_t g = *reinterpret_cast<const uint32_t*>(gate + t * a.ldp + col);
          const uint32_t wv = *reinterpret_cast<const uint32_t*>(w + col);
          const float f = inv * a.out_scale;
          *reinterpret_cast<uint32_t*>(out + t * a.ldo + col) =
              bf_pack(acc[j][m][y][2 * r] * f * bf_lo(wv) * silu_precise(bf_lo(g)),
                      acc[j][m][y][2 * r + 1] * f * bf_hi(wv) * silu_precise(bf_hi(g)));
        }
    }
}

template <int MT, int NJ>
cudaError_t launch_output(const ChunkParams& p, cudaStream_t st) {
  const int bytes = out_smem(p.a.dkp, p.a.dvp).total;
  auto kern = gla_chunk_output_kernel<MT, NJ>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  return launch_kernel(kern, dim3(p.chunks, p.a.H, p.a.B), dim3(kThreads), bytes, st, p);
}

int chunk_count(int S) { return (S + kC - 1) / kC; }

}  // namespace

bool gla_chunk_supported(const LinearAttnParams& a) { return a.dkp <= 256 && a.dvp <= 256; }

size_t gla_chunk_workspace_bytes(const LinearAttnParams& a) {
  const size_t heads = static_cast<size_t>(a.B) * a.H * chunk_count(a.S);
  return heads * a.dkp * (static_cast<size_t>(a.dvp) + 1) * sizeof(float);
}

cudaError_t launch_gla_chunk(const LinearAttnParams& a, void* ws, cudaStream_t st) {
  if (a.B == 0 || a.S == 0) return cudaSuccess;
  ChunkParams p;
  p.a = a;
  p.chunks = chunk_count(a.S);
  p.u = static_cast<float*>(ws);
  p.total = p.u + static_cast<size_t>(a.B) * a.H * p.chunks * a.dkp * a.dvp;
  const dim3 grid(p.chunks, a.H, a.B);
  const int bytes = (2 * kC * (a.dkp + 8) + kC * (a.dvp + 8)) * 2 + kThreads * 4;
  cudaError_t e = cudaFuncSetAttribute(gla_chunk_update_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  e = launch_kernel(gla_chunk_update_kernel, grid, dim3(kThreads), bytes, st, p);
  if (e != cudaSuccess) return e;
  const long long n4 = static_cast<long long>(a.B) * a.H * a.dkp * a.dvp / 4;
  e = launch_kernel(gla_chunk_scan_kernel, dim3(static_cast<unsigned>((n4 + kThreads - 1) / kThreads)), dim3(kThreads),
                    0, st, p);
  if (e != cudaSuccess) return e;
  if (a.dvp <= 64) return launch_output<2, 1>(p, st);
  if (a.dvp <= 128) return launch_output<4, 1>(p, st);
  return launch_output<4, 2>(p, st);
}

}  // namespace cdeep

// Window attention of a prompt (or a portion of one) in bf16: several queries of one sequence per
// block, all heads together, products on the tensor cores.
//
// The heads' weights are mixed after the softmax, so the normalisers of all heads must be known
// before any weight can be used: a first pass over the keys finds them, a second one forms the
// weights, mixes them and accumulates the values.  Per key tile of the second pass
//
//   1. scores of every (head, 16 queries) unit; weight = exp2(score - bias - lse), split into two
//      bf16 parts (16 significant bits), to shared memory as [head][query][key]
//   2. mixed = talk x weights, a product over the heads for every (query, key): talk is bf16 as
//      stored, the two parts of the weights are the other operand, sums in fp32; the result
//      replaces the high parts
//   3. out_h += mixed_h V
//
// The distance bias is a table of one tile's distances per head, computed once per tile.  Keys come
// from the projection buffer (this call's tokens) or from the ring (earlier ones), one bulk copy per
// key and tile.
//
// Why warp-level products: with all heads of a query tile in flight, scores, mixed weights and
// outputs of H heads x vdim columns exceed the 512 columns of tensor memory for any useful tile,
// and the mixed weights must pass through registers of warps that see every head anyway.
#include "kernels.h"
#include "mma.cuh"
#include "ptx.cuh"
#include "window_attention.cuh"

namespace cdeep {

namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kMasked = -1e30f;

// one row of `bytes` (a multiple of 16; both addresses 16-byte aligned), completing on `bar`
__device__ __forceinline__ void bulk_copy(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                   smem_addr(dst)), "l"(src), "r"(bytes), "r"(smem_addr(bar))
               : "memory");
}

// HU: heads dealt to the warps (8, 16 or 32); MB: blocks of 16 queries; KT: keys per tile
template <int HU, int MB, int KT>
struct Tile {
  static constexpr int kHP = HU < 16 ? 16 : HU;          // heads padded for the mixing product
  static constexpr int kMQ = MB * 16;
  static constexpr int kRow = KT + 8;                    // elements between the queries of a head's weights
  static constexpr int kHead = kMQ * kRow + 8;           // elements between heads
  static constexpr int kBias = kMQ + KT;                 // distances of a tile (one unused)
};

struct PrefillSmem {   // byte offsets
  int q, k, v, p, bias, stat, talk, r, total;
};
template <int HU, int MB, int KT, int DQ>
__host__ __device__ inline PrefillSmem prefill_smem(int H, int G, int dp, int vp) {
  using L = Tile<HU, MB, KT>;
  constexpr int HP = L::kHP;
  PrefillSmem s;
  const int kv = G * (dp > vp ? dp : vp) + 8;            // both buffers can hold a K tile (first pass)
  s.q = 0;                                               // [MQ][H * dp + 8] (DQ = 0)
  s.k = s.q + (DQ ? 0 : L::kMQ * (H * dp + 8) * 2);      // [KT][G * dp + 8]
  s.v = s.k + KT * kv * 2;                               // [KT][G * vp + 8]
  s.p = s.v + KT * kv * 2;                               // high parts, low parts: [HP][MQ][KT]
  s.bias = s.p + 2 * HP * L::kHead * 2;                  // [2][H][MQ + KT]
  s.stat = s.bias + 2 * H * L::kBias * 4;                // [H][MQ] log2 of the normaliser
  s.talk = s.stat + ((H * L::kMQ * 4 + 15) & ~15);       // [HP][HP + 8] bf16
  s.r = s.talk + HP * (HP + 8) * 2;                      // r1, r2 of the heads
  s.total = s.r + 2 * H * 4;
  return s;
}

// NV8: value columns / 8 at most; DQ: the queries stay in registers as DQ fragments (head width up to
// 16 DQ), 0: in shared memory; kExact: heads, head width and value columns are exactly HU, 16 DQ and
// 8 NV8, so that the products of a tile form straight-line code
template <int kWarps, int HU, int MB, int NV8, int KT, int DQ, bool kExact>
__global__ void __launch_bounds__(kWarps * 32, 1)
window_prefill_kernel(const WindowAttnParams p, int* status) {
  constexpr int kThreads = kWarps * 32;
  using L = Tile<HU, MB, KT>;
  constexpr int HP = L::kHP;
  constexpr int kMQ = L::kMQ;
  constexpr int kUnits = HU * MB / kWarps;               // (head, query block) units per warp
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ uint64_t bars[2];                           // K buffer, V buffer
  __shared__ int abort_word;
  if (threadIdx.x == 0) {
    mbar_init(&bars[0], 1);
    mbar_init(&bars[1], 1);
    abort_word = 0;
    fence_barrier_init();
  }
  pdl_enter();
  __syncthreads();
  const int H = kExact ? HU : p.H, G = p.G, rep = H / G;
  const int dp = kExact ? DQ * 16 : p.dp, vp = kExact ? NV8 * 8 : p.vp;
  const PrefillSmem off = prefill_smem<HU, MB, KT, DQ>(H, G, dp, vp);
  bf16* sQ = reinterpret_cast<bf16*>(smem + off.q);
  bf16* sK = reinterpret_cast<bf16*>(smem + off.k);
  bf16* sV = reinterpret_cast<bf16*>(smem + off.v);
  bf16* sP = reinterpret_cast<bf16*>(smem + off.p);
  bf16* sPl = sP + HP * L::kHead;
  float* sBias = reinterpret_cast<float*>(smem + off.bias);
  float* sStat = reinterpret_cast<float*>(smem + off.stat);
  bf16* sT = reinterpret_cast<bf16*>(smem + off.talk);
  float* sR = reinterpret_cast<float*>(smem + off.r);
  const int ldq = H * dp + 8, ldk = G * dp + 8, ldv = G * vp + 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = blockIdx.y;
  const int tile = gridDim.x - 1 - blockIdx.x;           // late tiles (more keys) first
  const int t0 = tile * kMQ;
  const int pos0 = window_pos0(p);
  const int i0 = pos0 + t0;                              // position of the tile's first query
  const int nq = min(kMQ, p.S - t0);
  const int i_last = i0 + nq - 1;
  const WindowKeys keys(i0, p.window, p.keep);
  const int kept_tiles = (keys.kept + KT - 1) / KT;
  const int tiles = kept_tiles + (i_last - keys.first + KT) / KT;
  const long long slots = p.keep + p.window;
  const bf16* ring_k = static_cast<const bf16*>(p.ring_k) + b * slots * G * dp;
  const bf16* ring_v = static_cast<const bf16*>(p.ring_v) + b * slots * G * vp;
  const long long row0 = static_cast<long long>(b) * p.S;
  const bf16* new_q = static_cast<const bf16*>(p.q) + row0 * p.ldp;
  const bf16* new_k = static_cast<const bf16*>(p.k) + row0 * p.ldp;
  const bf16* new_v = static_cast<const bf16*>(p.v) + row0 * p.ldp;

  // first position and number of keys of a tile
  auto tile_keys = [&](int t, int& j0, int& n) {
    if (t < kept_tiles) {
      j0 = t * KT;
      n = min(KT, keys.kept - j0);
    } else {
      j0 = keys.first + (t - kept_tiles) * KT;
      n = min(KT, i_last + 1 - j0);
    }
  };
  // Every warp issues its share of the keys, a lane per key; rows past the tile's keys repeat the last
  // one (their scores are masked, their weights zero).  Called with every thread done with the buffer.
  constexpr int kRowsWarp = KT / kWarps > 0 ? KT / kWarps : 1;
  auto load_tile = [&](int t, bf16* dst, int ld, const bf16* fresh, const bf16* ring, int width, uint64_t* bar) {
    const int r = warp * kRowsWarp + lane;
    if (t >= tiles || lane >= kRowsWarp || r >= KT) return;
    if (r == 0) mbar_arrive_expect_tx(bar, static_cast<uint32_t>(KT * width * 2));
    int j0, n;
    tile_keys(t, j0, n);
    const int j = j0 + min(r, n - 1);
    const bf16* src = fresh + (j - pos0) * p.ldp;
    if (j < pos0) src = ring + static_cast<long long>(window_slot(j, p.window, p.keep)) * width;
    bulk_copy(dst + r * ld, src, static_cast<uint32_t>(width * 2), bar);
  };
  volatile int* abort_flag = &abort_word;
  // use `count` (from 0) of a buffer has arrived
  auto wait_tile = [&](uint64_t* bar, int count) { mbar_wait(bar, static_cast<uint32_t>(count & 1), abort_flag); };
  auto fill_bias = [&](int t) {
    int j0, n;
    tile_keys(t, j0, n);
    float* dst = sBias + (t & 1) * H * L::kBias;
    for (int idx = tid; idx < H * L::kBias; idx += kThreads) {
      const int h = idx / L::kBias;
      const int d = max(i0 - j0 + (idx - h * L::kBias) - (KT - 1), 0);
      // r1 ln(1 + r2 d) in the log2 domain; its absolute error is that of the logarithm's argument
      dst[idx] = sR[h] * log2_approx(fmaf(sR[H + h], static_cast<float>(d), 1.0f));
    }
  };

  // ---------------------------------------------------------------- set-up
  uint32_t qf[kUnits][DQ ? DQ : 1][4];                  // A fragments of this warp's queries
  if constexpr (DQ > 0) {
#pragma unroll
    for (int u = 0; u < kUnits; ++u) {
      const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
#pragma unroll
      for (int x = 0; x < DQ; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = mb * 16 + (lane >> 2) + (e & 1) * 8, c = x * 16 + (lane & 3) * 2 + (e >> 1) * 8;
          qf[u][x][e] = (h < H && r < nq && c < dp)
                            ? *reinterpret_cast<const uint32_t*>(new_q + (t0 + r) * p.ldp + static_cast<long long>(h) * dp + c)
                            : 0u;
        }
    }
  } else {
    for (int r = warp; r < kMQ; r += kWarps)
      for (int c = lane * 8; c < H * dp; c += 256) {
        if (r < nq) copy16_async(sQ + r * ldq + c, new_q + (t0 + r) * p.ldp + c);
        else *reinterpret_cast<uint4*>(sQ + r * ldq + c) = make_uint4(0, 0, 0, 0);
      }
  }
  load_tile(0, sK, ldk, new_k, ring_k, G * dp, &bars[0]);
  for (int h = tid; h < H; h += kThreads) {
    sR[h] = to_f32(static_cast<const bf16*>(p.r1)[h]);
    sR[H + h] = to_f32(static_cast<const bf16*>(p.r2)[h]);
  }
  for (int idx = tid; idx < HP * HP; idx += kThreads) {
    const int h = idx / HP, g = idx - h * HP;
    sT[h * (HP + 8) + g] = (h < H && g < H) ? static_cast<const bf16*>(p.talk)[h * H + g] : __float2bfloat16_rn(0.f);
  }
  // weights of heads that do not exist stay zero
  for (int idx = tid; idx < (HP - H) * L::kHead / 8; idx += kThreads) {
    reinterpret_cast<uint4*>(sP + H * L::kHead)[idx] = make_uint4(0, 0, 0, 0);
    reinterpret_cast<uint4*>(sPl + H * L::kHead)[idx] = make_uint4(0, 0, 0, 0);
  }

  int key_head[kUnits];
#pragma unroll
  for (int u = 0; u < kUnits; ++u) key_head[u] = min((warp * kUnits + u) / MB, H - 1) / rep;
  const float scale2 = p.scale * kLog2e;
  const int r_lo = lane >> 2, c_lo = (lane & 3) * 2;     // row and column of a fragment's first element

  // scores of all units of this warp on 16 keys (from `k0` on) of the K tile in `kbuf` (scaled, biased,
  // masked, log2 domain)
  auto scores = [&](int t, int k0, const bf16* kbuf, float (&s)[kUnits][2][4]) {
    int j0, n;
    tile_keys(t, j0, n);
#pragma unroll
    for (int u = 0; u < kUnits; ++u)
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[u][nt][e] = 0.f;
    const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;   // B: 16 keys x 16
    const uint32_t k_base = smem_addr(kbuf + (k0 + b_row) * ldk + b_col);
    auto step = [&](int d, auto query) {                 // 16 elements of the head from d on
      uint32_t kb[4];
      int loaded = -1;
#pragma unroll
      for (int u = 0; u < kUnits; ++u) {
        const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
        if (!kExact && h >= H) break;
        const int c = key_head[u];
        if (u == 0 || c != loaded) {
          ldsm4(kb, k_base + static_cast<uint32_t>((c * dp + d) * 2));
          loaded = c;
        }
        uint32_t qa[4];
        query(u, h, mb, qa);
        mma16816(s[u][0], qa, kb[0], kb[1]);
        mma16816(s[u][1], qa, kb[2], kb[3]);
      }
    };
    if constexpr (DQ > 0) {
#pragma unroll
      for (int x = 0; x < DQ; ++x)
        if (kExact || x * 16 < dp)
          step(x * 16, [&](int u, int, int, uint32_t (&qa)[4]) {
#pragma unroll
            for (int e = 0; e < 4; ++e) qa[e] = qf[u][x][e];
          });
    } else {
      const uint32_t q_base = smem_addr(sQ + (lane & 15) * ldq + (lane >> 4) * 8);
      for (int d = 0; d < dp; d += 16)
        step(d, [&](int, int h, int mb, uint32_t (&qa)[4]) {
          ldsm4(qa, q_base + static_cast<uint32_t>((mb * 16 * ldq + h * dp + d) * 2));
        });
    }
    // every (query, key) of the tile visible?
    const bool full = n == KT && j0 + KT - 1 <= i0 && (i0 + kMQ - 1 - j0 < p.window || j0 + KT - 1 < p.keep);
#pragma unroll
    for (int u = 0; u < kUnits; ++u) {
      const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
      if (!kExact && h >= H) break;
      const float* bias = sBias + (t & 1) * H * L::kBias + h * L::kBias + KT - 1;
      if (full) {
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
            s[u][nt][e] = fmaf(s[u][nt][e], scale2,
                               -bias[mb * 16 + r_lo + (e >> 1) * 8 - (k0 + nt * 8 + c_lo + (e & 1))]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int qr = mb * 16 + r_lo + (e >> 1) * 8, kc = k0 + nt * 8 + c_lo + (e & 1);
            const int i = i0 + qr, j = j0 + kc;
            const bool seen = kc < n && j <= i && (i - j < p.window || j < p.keep);
            s[u][nt][e] = seen ? fmaf(s[u][nt][e], scale2, -bias[qr - kc]) : kMasked;
          }
      }
    }
  };

  // ---------------------------------------------------------------- first pass: normalisers
  float m_run[kUnits][2], l_run[kUnits][2];
#pragma unroll
  for (int u = 0; u < kUnits; ++u) {
    m_run[u][0] = m_run[u][1] = kMasked;
    l_run[u][0] = l_run[u][1] = 0.f;
  }
  copy_wait<0>();
  __syncthreads();                          // queries (when staged), talk, r1, r2 are written
  for (int t = 0; t < tiles; ++t) {
    fill_bias(t);
    wait_tile(&bars[t & 1], t >> 1);
    __syncthreads();                        // tile t is there; everybody is done with tile t - 1
    const bf16* kbuf = (t & 1) ? sV : sK;
    load_tile(t + 1, (t & 1) ? sK : sV, ldk, new_k, ring_k, G * dp, &bars[(t + 1) & 1]);
#pragma unroll
    for (int k0 = 0; k0 < KT; k0 += 16) {
      float s[kUnits][2][4];
      scores(t, k0, kbuf, s);
#pragma unroll
      for (int u = 0; u < kUnits; ++u) {
        if (!kExact && (warp * kUnits + u) / MB >= H) break;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const float m = fmaxf(fmaxf(m_run[u][r], fmaxf(s[u][0][2 * r], s[u][0][2 * r + 1])),
                                fmaxf(s[u][1][2 * r], s[u][1][2 * r + 1]));
          float l = l_run[u][r] * exp2_approx(m_run[u][r] - m);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) l += exp2_approx(s[u][nt][2 * r] - m) + exp2_approx(s[u][nt][2 * r + 1] - m);
          m_run[u][r] = m;
          l_run[u][r] = l;
        }
      }
    }
  }
  // merge the four lanes of a row (a lane that saw only masked keys drops out: exp2 of a huge negative)
#pragma unroll
  for (int u = 0; u < kUnits; ++u) {
    const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
    if (!kExact && h >= H) break;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float m = m_run[u][r], l = l_run[u][r];
#pragma unroll
      for (int x = 1; x < 4; x <<= 1) {
        const float mo = __shfl_xor_sync(0xffffffffu, m, x), lo = __shfl_xor_sync(0xffffffffu, l, x);
        const float mn = fmaxf(m, mo);
        l = l * exp2_approx(m - mn) + lo * exp2_approx(mo - mn);
        m = mn;
      }
      if ((lane & 3) == 0) sStat[h * kMQ + mb * 16 + r_lo + r * 8] = m + log2f(l);
    }
  }

  // ---------------------------------------------------------------- second pass
  float acc[kUnits][NV8][4];
#pragma unroll
  for (int u = 0; u < kUnits; ++u)
#pragma unroll
    for (int x = 0; x < NV8; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u][x][e] = 0.f;
  __syncthreads();                          // the first pass is done with both buffers; sStat is written
  load_tile(0, sK, ldk, new_k, ring_k, G * dp, &bars[0]);
  load_tile(0, sV, ldv, new_v, ring_v, G * vp, &bars[1]);
  const int k_uses = (tiles + 1) / 2, v_uses = tiles / 2;   // of the buffers in the first pass
  // talk as the A operand, kept in registers
  uint32_t ta[HP / 16][HP / 16][4];
#pragma unroll
  for (int x = 0; x < HP / 16; ++x)
#pragma unroll
    for (int y = 0; y < HP / 16; ++y)
      ldsm4(ta[x][y], smem_addr(sT + (x * 16 + (lane & 15)) * (HP + 8) + y * 16 + (lane >> 4) * 8));

  for (int t = 0; t < tiles; ++t) {
    fill_bias(t);
    wait_tile(&bars[0], k_uses + t);
    __syncthreads();
#pragma unroll 1
    for (int k0 = 0; k0 < KT; k0 += 16) {
      float s[kUnits][2][4];
      scores(t, k0, sK, s);
#pragma unroll
      for (int u = 0; u < kUnits; ++u) {
        const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
        if (!kExact && h >= H) break;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int qr = mb * 16 + r_lo + r * 8;
          const float lse = sStat[h * kMQ + qr];
          const int at = h * L::kHead + qr * L::kRow + k0 + c_lo;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const float a = s[u][nt][2 * r], c = s[u][nt][2 * r + 1];
            const float pa = exp2_approx(a - lse), pc = exp2_approx(c - lse);   // masked: 0
            uint32_t hi, lo;
            split_pair(pa, pc, hi, lo);
            *reinterpret_cast<uint32_t*>(sP + at + nt * 8) = hi;
            *reinterpret_cast<uint32_t*>(sPl + at + nt * 8) = lo;
          }
        }
      }
    }
    __syncthreads();
    load_tile(t + 1, sK, ldk, new_k, ring_k, G * dp, &bars[0]);
    // mix the heads: a warp takes 16 keys of one query at a time
#pragma unroll
    for (int it = 0; it < kMQ * (KT / 16) / kWarps; ++it) {
      const int item = it * kWarps + warp;
      const int qr = item / (KT / 16), k0 = (item - qr * (KT / 16)) * 16;
      float d[HP / 16][2][4];
#pragma unroll
      for (int x = 0; x < HP / 16; ++x)
#pragma unroll
        for (int y = 0; y < 2; ++y)
#pragma unroll
          for (int e = 0; e < 4; ++e) d[x][y][e] = 0.f;
      const int src = (lane & 15) * L::kHead + qr * L::kRow + k0 + (lane >> 4) * 8;
#pragma unroll
      for (int y = 0; y < HP / 16; ++y) {
        uint32_t bh[4], bl[4];
        ldsm4_t(bh, smem_addr(sP + src + y * 16 * L::kHead));
        ldsm4_t(bl, smem_addr(sPl + src + y * 16 * L::kHead));
#pragma unroll
        for (int x = 0; x < HP / 16; ++x) {
          mma16816(d[x][0], ta[x][y], bl[0], bl[1]);
          mma16816(d[x][1], ta[x][y], bl[2], bl[3]);
          mma16816(d[x][0], ta[x][y], bh[0], bh[1]);
          mma16816(d[x][1], ta[x][y], bh[2], bh[3]);
        }
      }
      __syncwarp();                         // every lane has read the old values
#pragma unroll
      for (int x = 0; x < HP / 16; ++x)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int h = x * 16 + r_lo + r * 8;
          if (h < H) {
            bf16* dst = sP + h * L::kHead + qr * L::kRow + k0 + c_lo;
            *reinterpret_cast<uint32_t*>(dst) = bf_pack(d[x][0][2 * r], d[x][0][2 * r + 1]);
            *reinterpret_cast<uint32_t*>(dst + 8) = bf_pack(d[x][1][2 * r], d[x][1][2 * r + 1]);
          }
        }
    }
    wait_tile(&bars[1], v_uses + t);
    __syncthreads();
    // out_h += mixed_h V_c
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t pa[kUnits][4];
#pragma unroll
      for (int u = 0; u < kUnits; ++u) {
        const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
        if (kExact || h < H)
          ldsm4(pa[u], smem_addr(sP + h * L::kHead + (mb * 16 + (lane & 15)) * L::kRow + kk * 16 + (lane >> 4) * 8));
      }
      const uint32_t v_base = smem_addr(sV + (kk * 16 + (lane & 15)) * ldv + (lane >> 4) * 8);
#pragma unroll
      for (int x = 0; x < NV8 / 2; ++x) {
        if (kExact || x * 16 < vp) {
          uint32_t vb[4];
          int loaded = -1;
#pragma unroll
          for (int u = 0; u < kUnits; ++u) {
            if (!kExact && (warp * kUnits + u) / MB >= H) break;
            const int c = key_head[u];
            if (u == 0 || c != loaded) {
              ldsm4_t(vb, v_base + static_cast<uint32_t>((c * vp + x * 16) * 2));
              loaded = c;
            }
            mma16816(acc[u][2 * x], pa[u], vb[0], vb[1]);
            mma16816(acc[u][2 * x + 1], pa[u], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();
    load_tile(t + 1, sV, ldv, new_v, ring_v, G * vp, &bars[1]);
  }
  if (tid == 0 && *abort_flag) atomicExch(status, 1);

  bf16* out = static_cast<bf16*>(p.out);
#pragma unroll
  for (int u = 0; u < kUnits; ++u) {
    const int unit = warp * kUnits + u, h = unit / MB, mb = unit - h * MB;
    if (!kExact && h >= H) break;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int qr = mb * 16 + r_lo + r * 8;
      if (qr >= nq) continue;
      bf16* orow = out + (row0 + t0 + qr) * p.ldo + static_cast<long long>(h) * vp + c_lo;
#pragma unroll
      for (int x = 0; x < NV8; ++x)
        if (x * 8 < vp)
          *reinterpret_cast<uint32_t*>(orow + x * 8) = bf_pack(acc[u][x][2 * r] * p.out_scale, acc[u][x][2 * r + 1] * p.out_scale);
    }
  }
}

constexpr int kMaxDynSmem = 226 * 1024;

template <int W, int HU, int MB, int NV8, int KT, int DQ, bool kExact = false>
bool try_launch(const WindowAttnParams& p, cudaStream_t st, cudaError_t& e, bool only_ask) {
  const int bytes = prefill_smem<HU, MB, KT, DQ>(p.H, p.G, p.dp, p.vp).total;
  if (bytes > kMaxDynSmem || p.H > HU || p.vp > NV8 * 8 || (DQ && p.dp > DQ * 16)) return false;
  if (kExact && (p.H != HU || p.vp != NV8 * 8 || p.dp != DQ * 16)) return false;
  if (only_ask) return true;
  auto kern = window_prefill_kernel<W, HU, MB, NV8, KT, DQ, kExact>;
  e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem);
  if (e != cudaSuccess) return true;
  const int mq = MB * 16;
  e = launch_kernel(kern, dim3((p.S + mq - 1) / mq, p.B), dim3(W * 32), bytes, st, p, device_status_word());
  return true;
}

// Registers per thread bound units x (value columns + query fragments), shared memory the rest: the
// largest tile that fits.
bool dispatch(const WindowAttnParams& p, cudaStream_t st, cudaError_t& e, bool only_ask) {
  return (p.S > 16 && try_launch<16, 8, 2, 16, 32, 8, true>(p, st, e, only_ask)) ||
         try_launch<16, 16, 1, 16, 32, 8, true>(p, st, e, only_ask) ||
         (p.S > 16 && try_launch<16, 8, 2, 16, 32, 8>(p, st, e, only_ask)) ||
         try_launch<16, 16, 1, 16, 32, 8>(p, st, e, only_ask) ||
         try_launch<16, 16, 1, 16, 16, 0>(p, st, e, only_ask) ||
         try_launch<8, 8, 1, 32, 16, 0>(p, st, e, only_ask) ||
         try_launch<16, 32, 1, 8, 16, 0>(p, st, e, only_ask);
}

}  // namespace

bool window_prefill_supported(const WindowAttnParams& p) {
  cudaError_t e = cudaSuccess;
  return dispatch(p, nullptr, e, true);
}

cudaError_t launch_window_prefill(const WindowAttnParams& p, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  cudaError_t e = cudaSuccess;
  return dispatch(p, st, e, false) ? e : cudaErrorInvalidValue;
}

}  // namespace cdeep

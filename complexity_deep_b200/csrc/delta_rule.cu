// Delta rule with one decay per key channel: convolution and norms ahead of the recurrence, the
// token-by-token recurrence (any storage type), and the head norm and gate behind it.
#include "delta_rule.cuh"
#include "kernels.h"

namespace cdeep {

namespace {

constexpr int kThreads = 256;

// ---------------------------------------------------------------- convolution, silu, norms
// A warp takes `run` tokens of one head of q, k or v; a lane owns eight channels at a time.  The warp
// of the first run also moves the last inputs of the call into the ring, after it has read the earlier
// ones (run >= taps - 1: nobody else reads the ring).
template <typename T>
__global__ void __launch_bounds__(kThreads)
delta_prepare_kernel(const DeltaParams p, int run) {
  pdl_enter();
  const int lane = threadIdx.x & 31;
  const int slots = 2 * p.G + p.H, C = delta_channels(p);
  const int item = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5), b = blockIdx.y;
  const int slot = item % slots, t0 = item / slots * run;
  if (t0 >= p.S) return;
  const bool is_v = slot >= 2 * p.G;
  const int width = is_v ? p.dvp : p.dkp;
  const int col = is_v ? 2 * p.G * p.dkp + (slot - 2 * p.G) * p.dvp : slot * p.dkp;
  const T* src = static_cast<const T*>(is_v ? p.v : slot < p.G ? p.q : p.k) +
                 (is_v ? (slot - 2 * p.G) * p.dvp : (slot < p.G ? slot : slot - p.G) * p.dkp);
  const long long row0 = static_cast<long long>(b) * p.S;
  const T* taps = static_cast<const T*>(p.taps_w) + col;
  T* ring = static_cast<T*>(p.ring) + static_cast<long long>(b) * p.taps * C + col;
  T* act = static_cast<T*>(p.act) + col;
  const int pos0 = first_position(p);
  const float scale = slot < p.G ? 1.0f / sqrtf(static_cast<float>(p.dk)) : 1.0f;
  for (int t = t0; t < min(t0 + run, p.S); ++t) {
    float ss = 0.f;
    for (int c = lane * 8; c < width; c += 256) {
      float y[8] = {};
      for (int j = p.taps - 1; j >= 0; --j) {              // j tokens back
        const int pos = pos0 + t - j;
        if (pos < 0) continue;
        float x[8], w[8];
        if (t - j >= 0) load8(src + (row0 + t - j) * p.ldp + c, x);
        else load8(ring + static_cast<long long>(pos % p.taps) * C + c, x);
        load8(taps + static_cast<long long>(p.taps - 1 - j) * C + c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = fmaf(w[e], x[e], y[e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        y[e] = to_f32(from_f32<T>(silu_precise(y[e])));
        ss += y[e] * y[e];
      }
      store8(act + (row0 + t) * C + c, y);
    }
    if (!is_v) {
      ss = warp_add(ss);
      if (lane == 0) p.inv[(row0 + t) * 2 * p.G + slot] = scale / sqrtf(ss + 1e-6f);
    }
  }
  if (t0 == 0)
    for (int t = max(0, p.S - p.taps); t < p.S; ++t)
      for (int c = lane * 8; c < width; c += 256) {
        float x[8];
        load8(src + (row0 + t) * p.ldp + c, x);
        store8(ring + static_cast<long long>((pos0 + t) % p.taps) * C + c, x);
      }
}

// The usual sizes: up to four taps and heads up to 8 GL wide.  A group of GL lanes takes kRun tokens of one
// head; a lane's eight channels of all of them are loaded up front and pass through a window in registers.
constexpr int kRun = 8;
constexpr int kWindow = 4;

template <typename T, int GL>
__global__ void __launch_bounds__(kThreads)
delta_prepare_window_kernel(const DeltaParams p) {
  pdl_enter();
  const int slots = 2 * p.G + p.H, C = delta_channels(p), b = blockIdx.y;
  const int runs = (p.S + kRun - 1) / kRun;
  const int item = (blockIdx.x * kThreads + threadIdx.x) / GL, c = (threadIdx.x % GL) * 8;
  const bool live = item < runs * slots;                    // idle groups stay for the shuffles
  const int slot = live ? item % slots : 0, t0 = live ? item / slots * kRun : p.S;
  const bool is_v = slot >= 2 * p.G;
  const int width = is_v ? p.dvp : p.dkp;
  const bool ok = live && c < width;
  const int col = (is_v ? 2 * p.G * p.dkp + (slot - 2 * p.G) * p.dvp : slot * p.dkp) + c;
  const T* src = static_cast<const T*>(is_v ? p.v : slot < p.G ? p.q : p.k) +
                 (is_v ? (slot - 2 * p.G) * p.dvp : (slot < p.G ? slot : slot - p.G) * p.dkp) + c;
  const long long row0 = static_cast<long long>(b) * p.S;
  const T* taps = static_cast<const T*>(p.taps_w) + col;
  T* ring = static_cast<T*>(p.ring) + static_cast<long long>(b) * p.taps * C + col;
  const int pos0 = first_position(p);
  Raw8<T> raw[kRun + kWindow - 1] = {};                     // tokens t0 - 3 ...
#pragma unroll
  for (int x = 0; x < kRun + kWindow - 1; ++x) {
    const int t = t0 + x - (kWindow - 1);
    if (!ok || t >= p.S || pos0 + t < 0) continue;
    if (t >= 0) raw_load(src + (row0 + t) * p.ldp, raw[x]);
    else if (-t < p.taps) raw_load(ring + static_cast<long long>((pos0 + t) % p.taps) * C, raw[x]);
  }
  float w[kWindow][8] = {};                                 // w[j]: j tokens back
#pragma unroll
  for (int j = 0; j < kWindow; ++j)
    if (ok && j < p.taps) load8(taps + static_cast<long long>(p.taps - 1 - j) * C, w[j]);
  float win[kWindow][8] = {};
#pragma unroll
  for (int x = 0; x < kWindow - 1; ++x) raw_unpack(raw[x], win[(x + 1) % kWindow]);
  const float scale = slot < p.G ? 1.0f / sqrtf(static_cast<float>(p.dk)) : 1.0f;
#pragma unroll
  for (int x = 0; x < kRun; ++x) {
    const int t = t0 + x;                                   // its input goes to window slot x % 4
    raw_unpack(raw[x + kWindow - 1], win[x % kWindow]);
    float y[8] = {}, ss = 0.f;
#pragma unroll
    for (int j = kWindow - 1; j >= 0; --j)
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = fmaf(w[j][e], win[(x - j + kWindow) % kWindow][e], y[e]);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      y[e] = to_f32(from_f32<T>(sizeof(T) == 2 ? silu_fast(y[e]) : silu_precise(y[e])));
      ss += y[e] * y[e];
    }
#pragma unroll
    for (int o = GL / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (ok && t < p.S) {
      store8(static_cast<T*>(p.act) + (row0 + t) * C + col, y);
      if (!is_v && c == 0) p.inv[(row0 + t) * 2 * p.G + slot] = scale / sqrtf(ss + 1e-6f);
    }
  }
  if (ok && t0 == 0)
    for (int t = max(0, p.S - p.taps); t < p.S; ++t) {
      float x[8];
      load8(src + (row0 + t) * p.ldp, x);
      store8(ring + static_cast<long long>((pos0 + t) % p.taps) * C, x);
    }
}

// ---------------------------------------------------------------- token by token
constexpr int kSteps = 16;     // tokens staged in shared memory at a time
constexpr int kCols = 32;      // state columns per block, four per warp

// A lane owns M rows (lane % 8, + 8, ...) of one column of the state (dkp <= 8 M).
template <typename T, int M>
__global__ void __launch_bounds__(kThreads)
delta_sequence_kernel(const DeltaParams p) {
  extern __shared__ float sm[];
  pdl_enter();
  const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dkp = p.dkp, dvp = p.dvp, C = delta_channels(p);
  float* sq = sm;                          // [kSteps][dkp]
  float* sk = sq + kSteps * dkp;
  float* sa = sk + kSteps * dkp;           // decays
  float* sv = sa + kSteps * dkp;           // [kSteps][kCols]
  float* sb = sv + kSteps * kCols;         // [kSteps] beta
  float* sx = sb + kSteps;                 // [kSteps] k . q
  const int cl = warp * 4 + (lane >> 3), r0 = lane & 7, col = blockIdx.x * kCols + cl;
  const bool col_ok = col < dvp;
  float* S = p.state + (static_cast<long long>(b) * p.H + h) * dkp * dvp + col;
  float s[M];
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int r = r0 + 8 * m;
    s[m] = (r < dkp && col_ok) ? S[static_cast<long long>(r) * dvp] : 0.f;
  }
  const long long row0 = static_cast<long long>(b) * p.S;
  const float rate = p.rate[h];
  for (int t0 = 0; t0 < p.S; t0 += kSteps) {
    const int n = min(kSteps, p.S - t0);
    for (int idx = tid; idx < n * dkp; idx += kThreads) {
      const int t = idx / dkp, c = idx - t * dkp;
      const long long row = row0 + t0 + t;
      const T* act = static_cast<const T*>(p.act) + row * C;
      const float* inv = p.inv + row * 2 * p.G;
      sq[idx] = to_f32(act[g * dkp + c]) * inv[g];
      sk[idx] = to_f32(act[(p.G + g) * dkp + c]) * inv[p.G + g];
      sa[idx] = expf(-rate * softplus_precise(p.zg[row * p.ldz + h * dkp + c] + p.dt_bias[h * dkp + c]));
    }
    for (int idx = tid; idx < n * kCols; idx += kThreads) {
      const int t = idx / kCols, c = blockIdx.x * kCols + idx - t * kCols;
      sv[idx] = c < dvp ? to_f32(static_cast<const T*>(p.act)[(row0 + t0 + t) * C + 2 * p.G * dkp + h * dvp + c]) : 0.f;
    }
    for (int t = tid; t < n; t += kThreads)
      sb[t] = sigmoid_precise(to_f32(static_cast<const T*>(p.b)[(row0 + t0 + t) * p.ldp + h]));
    __syncthreads();
    for (int t = warp; t < n; t += kThreads / 32) {
      float x = 0.f;
      for (int c = lane; c < dkp; c += 32) x += sk[t * dkp + c] * sq[t * dkp + c];
      x = warp_add(x);
      if (lane == 0) sx[t] = x;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      float a = 0.f, o = 0.f;
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int r = r0 + 8 * m;
        if (r < dkp) {
          s[m] *= sa[t * dkp + r];
          a = fmaf(s[m], sk[t * dkp + r], a);
          o = fmaf(s[m], sq[t * dkp + r], o);
        }
      }
#pragma unroll
      for (int d = 1; d < 8; d <<= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, d);
        o += __shfl_xor_sync(0xffffffffu, o, d);
      }
      const float u = sb[t] * (sv[t * kCols + cl] - a);
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int r = r0 + 8 * m;
        if (r < dkp) s[m] = fmaf(sk[t * dkp + r], u, s[m]);
      }
      if (r0 == 0 && col_ok)
        p.o_raw[(row0 + t0 + t) * (p.H * dvp) + static_cast<long long>(h) * dvp + col] = fmaf(sx[t], u, o);
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int r = r0 + 8 * m;
    if (r < dkp && col_ok) S[static_cast<long long>(r) * dvp] = s[m];
  }
}

// ---------------------------------------------------------------- one token
// Sums of N values over the block; every thread gets them (a barrier on both sides)
template <int N>
__device__ __forceinline__ void block_add(float (&v)[N], float* s) {
#pragma unroll
  for (int x = 0; x < N; ++x) v[x] = warp_add(v[x]);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) {
#pragma unroll
    for (int x = 0; x < N; ++x) s[x * (kThreads / 32) + (threadIdx.x >> 5)] = v[x];
  }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < N; ++x) {
    v[x] = 0.f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) v[x] += s[x * (kThreads / 32) + w];
  }
}

// One of the values that a step needs before its recurrence: a channel of q, k or v after convolution and
// silu, or a decay.  Loaded before it is used, so that a thread has several on the way.
template <typename T>
struct StepItem {
  T x[kWindow], w[kWindow];
  float z;
};

// A block per head and sequence does the whole step: convolution, norms, decay, recurrence, head norm,
// gate.  A thread keeps RP rows of four columns of the state in registers (loaded before anything
// else), so the state is read and written once: with a = (g S)^T k and o = (g S)^T q from one pass,
// u = beta (v - a), the new state is g S + k u^T and the result o + (k . q) u.
template <typename T, int RP>
__global__ void __launch_bounds__(kThreads, RP <= 16 ? 2 : 1)
delta_step_kernel(const DeltaParams p) {
  extern __shared__ float sm[];
  __shared__ float s_red[3 * kThreads / 32];
  pdl_enter();
  const int h = blockIdx.x, b = blockIdx.y, rep = p.H / p.G, g = h / rep, tid = threadIdx.x;
  const int dkp = p.dkp, dvp = p.dvp, C = delta_channels(p);
  float* sq = sm;                  // [dkp]
  float* sk = sq + dkp;
  float* sg = sk + dkp;            // decays
  float* sv = sg + dkp;            // [dvp] v, then u
  float* so = sv + dvp;            // [dvp] result
  float* sp = so + dvp;            // [2][row groups][dvp] partial sums
  const int cgs = dvp / 4, rgs = kThreads / cgs, rg = tid / cgs, col = (tid - rg * cgs) * 4;
  const bool live = rg < rgs;
  float* S = p.state + (static_cast<long long>(b) * p.H + h) * dkp * dvp + col;
  float4 s[RP];
#pragma unroll
  for (int m = 0; m < RP; ++m) {
    const int r = rg + m * rgs;
    s[m] = (live && r < dkp) ? *reinterpret_cast<const float4*>(S + static_cast<long long>(r) * dvp)
                             : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int pos = first_position(p);
  T* ring = static_cast<T*>(p.ring) + static_cast<long long>(b) * p.taps * C;
  const T* taps = static_cast<const T*>(p.taps_w);
  int back[kWindow];                      // offset in the ring of the input j tokens back, -1: none
#pragma unroll
  for (int j = 0; j < kWindow; ++j) back[j] = j < p.taps && j <= pos ? (pos - j) % p.taps * C : -1;
  const bool first = h % rep == 0;        // the block that brings the ring up to date for its q / k head
  const float rate = p.rate[h];
  const float* zg = p.zg + b * p.ldz;
  // items: q, k, v channels, decays
  const int n_k = dkp, n_v = 2 * dkp, n_g = n_v + dvp, total = n_g + dkp;
  auto channel_of = [&](int i) { return i < n_v ? (i < n_k ? g * dkp + i : (p.G + g) * dkp + i - n_k) : 2 * p.G * dkp + h * dvp + i - n_v; };
  auto load = [&](int i, StepItem<T>& r) {
    if (i >= total) return;
    if (i >= n_g) {
      const int c = h * dkp + i - n_g;
      r.z = zg[c] + p.dt_bias[c];
      return;
    }
    const T* in = i < n_k ? static_cast<const T*>(p.q) + g * dkp + i
                          : i < n_v ? static_cast<const T*>(p.k) + g * dkp + i - n_k
                                    : static_cast<const T*>(p.v) + h * dvp + i - n_v;
    const int ch = channel_of(i);
    r.x[0] = in[b * p.ldp];
    r.w[0] = taps[(p.taps - 1) * C + ch];
#pragma unroll
    for (int j = 1; j < kWindow; ++j) {
      r.x[j] = back[j] >= 0 ? ring[back[j] + ch] : from_f32<T>(0.f);
      r.w[j] = back[j] >= 0 ? taps[(p.taps - 1 - j) * C + ch] : from_f32<T>(0.f);
    }
  };
  auto finish = [&](int i, const StepItem<T>& r) {
    if (i >= total) return;
    if (i >= n_g) {
      sg[i - n_g] = sizeof(T) == 2 ? exp2_approx(-rate * 1.4426950408889634f * softplus_fast(r.z))
                                   : expf(-rate * softplus_precise(r.z));
      return;
    }
    const int ch = channel_of(i);
    float y = 0.f;
    for (int j = p.taps - 1; j >= kWindow; --j)             // more taps than the window holds
      if (j <= pos)
        y = fmaf(to_f32(taps[(p.taps - 1 - j) * C + ch]), to_f32(ring[(pos - j) % p.taps * C + ch]), y);
#pragma unroll
    for (int j = kWindow - 1; j >= 0; --j) y = fmaf(to_f32(r.w[j]), to_f32(r.x[j]), y);
    y = to_f32(from_f32<T>(sizeof(T) == 2 ? silu_fast(y) : silu_precise(y)));
    if (i < n_v) sq[i] = y;               // k follows q
    else sv[i - n_v] = y;
    if (i >= n_v || first) ring[back[0] + ch] = r.x[0];
  };
  for (int i = tid; i < total; i += 2 * kThreads) {
    StepItem<T> r0, r1;
    load(i, r0);
    load(i + kThreads, r1);
    finish(i, r0);
    finish(i + kThreads, r1);
  }
  __syncthreads();
  float sums[3] = {0.f, 0.f, 0.f};        // |q|^2, |k|^2, k . q
  for (int c = tid; c < dkp; c += kThreads) {
    const float q = sq[c], k = sk[c];
    sums[0] += q * q;
    sums[1] += k * k;
    sums[2] += k * q;
  }
  block_add(sums, s_red);
  const float iq = 1.0f / sqrtf(static_cast<float>(p.dk)) / sqrtf(sums[0] + 1e-6f), ik = 1.0f / sqrtf(sums[1] + 1e-6f);
  const float kq = sums[2] * iq * ik;
  const float beta = sigmoid_precise(to_f32(static_cast<const T*>(p.b)[b * p.ldp + h]));
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f), o = a;
  if (live) {
#pragma unroll
    for (int m = 0; m < RP; ++m) {
      const int r = rg + m * rgs;
      if (r < dkp) {
        const float f = sg[r], k = sk[r] * ik, q = sq[r] * iq;
        s[m].x *= f; s[m].y *= f; s[m].z *= f; s[m].w *= f;
        a.x = fmaf(s[m].x, k, a.x); a.y = fmaf(s[m].y, k, a.y); a.z = fmaf(s[m].z, k, a.z); a.w = fmaf(s[m].w, k, a.w);
        o.x = fmaf(s[m].x, q, o.x); o.y = fmaf(s[m].y, q, o.y); o.z = fmaf(s[m].z, q, o.z); o.w = fmaf(s[m].w, q, o.w);
      }
    }
    *reinterpret_cast<float4*>(sp + rg * dvp + col) = a;
    *reinterpret_cast<float4*>(sp + (rgs + rg) * dvp + col) = o;
  }
  __syncthreads();
  float ss[1] = {0.f};
  for (int c = tid; c < dvp; c += kThreads) {
    float x = 0.f, y = 0.f;
    for (int r = 0; r < rgs; ++r) {
      x += sp[r * dvp + c];
      y += sp[(rgs + r) * dvp + c];
    }
    const float u = beta * (sv[c] - x);
    sv[c] = u;
    y = fmaf(kq, u, y);
    so[c] = y;
    ss[0] += y * y;
  }
  block_add(ss, s_red);
  if (live) {
    const float4 u = *reinterpret_cast<const float4*>(sv + col);
#pragma unroll
    for (int m = 0; m < RP; ++m) {
      const int r = rg + m * rgs;
      if (r < dkp) {
        const float k = sk[r] * ik;
        s[m].x = fmaf(k, u.x, s[m].x); s[m].y = fmaf(k, u.y, s[m].y);
        s[m].z = fmaf(k, u.z, s[m].z); s[m].w = fmaf(k, u.w, s[m].w);
        *reinterpret_cast<float4*>(S + static_cast<long long>(r) * dvp) = s[m];
      }
    }
  }
  const float r = 1.0f / sqrtf(ss[0] / static_cast<float>(p.dv) + p.eps);
  T* out = static_cast<T*>(p.out) + b * p.ldo + static_cast<long long>(h) * dvp;
  for (int c = tid; c < dvp; c += kThreads)
    out[c] = from_f32<T>(so[c] * r * to_f32(static_cast<const T*>(p.norm_w)[c]) *
                         sigmoid_precise(zg[p.H * dkp + h * dvp + c]) * p.out_scale);
}

// ---------------------------------------------------------------- head norm and gate
// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(kThreads)
delta_finish_kernel(const DeltaParams p) {
  pdl_enter();
  const long long item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(p.B) * p.S * p.H) return;
  const int lane = threadIdx.x & 31;
  const long long row = item / p.H;
  const int h = static_cast<int>(item - row * p.H);
  const float* o = p.o_raw + item * p.dvp;
  const float* gate = p.zg + row * p.ldz + p.H * p.dkp + static_cast<long long>(h) * p.dvp;
  T* out = static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.dvp;
  float ss = 0.f;
  for (int c = lane; c < p.dvp; c += 32) ss += o[c] * o[c];
  const float r = 1.0f / sqrtf(warp_add(ss) / static_cast<float>(p.dv) + p.eps);
  for (int c = lane; c < p.dvp; c += 32)
    out[c] = from_f32<T>(o[c] * r * to_f32(static_cast<const T*>(p.norm_w)[c]) * sigmoid_precise(gate[c]) * p.out_scale);
}

// heads up to 8 GL wide: a group of GL lanes per (row, head), eight columns per lane
template <typename T, int GL>
__global__ void __launch_bounds__(kThreads)
delta_finish_group_kernel(const DeltaParams p) {
  pdl_enter();
  const long long items = static_cast<long long>(p.B) * p.S * p.H;
  const long long item = (static_cast<long long>(blockIdx.x) * kThreads + threadIdx.x) / GL;
  const int c = (threadIdx.x % GL) * 8;
  const bool ok = item < items && c < p.dvp;
  const long long row = ok ? item / p.H : 0;
  const int h = ok ? static_cast<int>(item - row * p.H) : 0;
  float o[8] = {}, gate[8] = {}, w[8] = {}, ss = 0.f;
  if (ok) {
    load8(p.o_raw + item * p.dvp + c, o);
    load8(p.zg + row * p.ldz + p.H * p.dkp + static_cast<long long>(h) * p.dvp + c, gate);
    load8(static_cast<const T*>(p.norm_w) + c, w);
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += o[e] * o[e];
#pragma unroll
  for (int d = GL / 2; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  const float r = p.out_scale / sqrtf(ss / static_cast<float>(p.dv) + p.eps);
#pragma unroll
  for (int e = 0; e < 8; ++e)
    o[e] *= r * w[e] * (sizeof(T) == 2 ? 1.0f / (1.0f + exp2_approx(-1.4426950408889634f * gate[e])) : sigmoid_precise(gate[e]));
  if (ok) store8(static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(h) * p.dvp + c, o);
}

template <typename T, int GL>
cudaError_t launch_window(const DeltaParams& p, cudaStream_t st) {
  const long long lanes = static_cast<long long>((p.S + kRun - 1) / kRun) * (2 * p.G + p.H) * GL;
  return launch_kernel(delta_prepare_window_kernel<T, GL>, dim3(static_cast<unsigned>((lanes + kThreads - 1) / kThreads), p.B),
                       dim3(kThreads), 0, st, p);
}

template <typename T, int GL>
cudaError_t launch_finish_group(const DeltaParams& p, cudaStream_t st) {
  const long long lanes = static_cast<long long>(p.B) * p.S * p.H * GL;
  return launch_kernel(delta_finish_group_kernel<T, GL>, dim3(static_cast<unsigned>((lanes + kThreads - 1) / kThreads)),
                       dim3(kThreads), 0, st, p);
}

template <typename T>
cudaError_t launch_finish(const DeltaParams& p, cudaStream_t st) {
  if (p.dvp <= 64) return launch_finish_group<T, 8>(p, st);
  if (p.dvp <= 128) return launch_finish_group<T, 16>(p, st);
  if (p.dvp <= 256) return launch_finish_group<T, 32>(p, st);
  const long long items = static_cast<long long>(p.B) * p.S * p.H;
  return launch_kernel(delta_finish_kernel<T>, dim3(static_cast<unsigned>((items + 7) / 8)), dim3(kThreads), 0, st, p);
}

template <typename T>
cudaError_t launch_prepare(const DeltaParams& p, cudaStream_t st) {
  const int widest = p.dkp > p.dvp ? p.dkp : p.dvp;
  if (p.taps <= kWindow) {
    if (widest <= 64) return launch_window<T, 8>(p, st);
    if (widest <= 128) return launch_window<T, 16>(p, st);
    if (widest <= 256) return launch_window<T, 32>(p, st);
  }
  const int run = p.taps > 9 ? p.taps - 1 : 8;
  const long long items = static_cast<long long>((p.S + run - 1) / run) * (2 * p.G + p.H);
  return launch_kernel(delta_prepare_kernel<T>, dim3(static_cast<unsigned>((items + 7) / 8), p.B), dim3(kThreads), 0, st,
                       p, run);
}

template <typename T, int M>
cudaError_t launch_sequence_m(const DeltaParams& p, cudaStream_t st) {
  const size_t bytes = (3 * kSteps * p.dkp + kSteps * kCols + 2 * kSteps) * sizeof(float);
  cudaError_t e = allow_smem<delta_sequence_kernel<T, M>>(static_cast<int>(bytes));
  if (e != cudaSuccess) return e;
  return launch_kernel(delta_sequence_kernel<T, M>, dim3((p.dvp + kCols - 1) / kCols, p.H, p.B), dim3(kThreads), bytes,
                       st, p);
}

template <typename T>
cudaError_t launch_sequence(const DeltaParams& p, cudaStream_t st) {
  if (p.dkp <= 32) return launch_sequence_m<T, 4>(p, st);
  if (p.dkp <= 64) return launch_sequence_m<T, 8>(p, st);
  if (p.dkp <= 128) return launch_sequence_m<T, 16>(p, st);
  if (p.dkp <= 256) return launch_sequence_m<T, 32>(p, st);
  if (p.dkp <= 512) return launch_sequence_m<T, 64>(p, st);
  return cudaErrorInvalidValue;
}

int step_rows(const DeltaParams& p) {       // rows of the state per thread
  const int rgs = kThreads / (p.dvp / 4);
  return rgs > 0 ? (p.dkp + rgs - 1) / rgs : 1 << 20;
}

template <typename T>
cudaError_t launch_step(const DeltaParams& p, cudaStream_t st) {
  const int rgs = kThreads / (p.dvp / 4), rp = step_rows(p);
  const size_t bytes = (3 * p.dkp + 2 * p.dvp + 2 * rgs * p.dvp) * sizeof(float);
  const dim3 grid(p.H, p.B), block(kThreads);
  if (rp <= 4) return launch_kernel(delta_step_kernel<T, 4>, grid, block, bytes, st, p);
  if (rp <= 8) return launch_kernel(delta_step_kernel<T, 8>, grid, block, bytes, st, p);
  if (rp <= 16) return launch_kernel(delta_step_kernel<T, 16>, grid, block, bytes, st, p);
  if (rp <= 32) return launch_kernel(delta_step_kernel<T, 32>, grid, block, bytes, st, p);
  return cudaErrorInvalidValue;
}

}  // namespace

bool delta_step_supported(const DeltaParams& p) {
  return p.S == 1 && p.dvp <= 4 * kThreads && step_rows(p) <= 32;
}

cudaError_t launch_delta_step(const DeltaParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0) return cudaSuccess;
  return fp32 ? launch_step<float>(p, st) : launch_step<bf16>(p, st);
}

bool delta_supported(const DeltaParams& p) { return p.dkp <= 512 && p.B <= 65535; }

cudaError_t launch_delta_prepare(const DeltaParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_prepare<float>(p, st) : launch_prepare<bf16>(p, st);
}

cudaError_t launch_delta_sequence(const DeltaParams& p, int fp32, cudaStream_t st) {
  if (p.B == 0 || p.S == 0) return cudaSuccess;
  return fp32 ? launch_sequence<float>(p, st) : launch_sequence<bf16>(p, st);
}

cudaError_t launch_delta_finish(const DeltaParams& p, int fp32, cudaStream_t st) {
  const long long items = static_cast<long long>(p.B) * p.S * p.H;
  if (items == 0) return cudaSuccess;
  return fp32 ? launch_finish<float>(p, st) : launch_finish<bf16>(p, st);
}

}  // namespace cdeep

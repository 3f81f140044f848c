// Kernels around a residual stream kept in fp32: embedding gather into the stream, RMSNorm or layer
// norm of a stream row into the operand type of the next product, and the 32-bit matrix product used
// when a model runs entirely in fp32 (no reduced-precision mode anywhere on that path).
#include "elem.cuh"
#include "kernels.h"

namespace cdeep {

namespace {

struct Positions {          // learned position vectors (table nullptr: none)
  const void* table;
  int P, S, pos0;
  const int* pos_dev;
};

// x[t, :] = table[ids[t], :] (+ the vector of the row's position) in fp32; columns [W, ldx) are zero.
// Ids outside the table are clamped to it (as in the dispatch kernels), and so are positions, so a
// bad id can never read out of bounds.
template <typename T>
__global__ void __launch_bounds__(128)
embed_rows_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const Positions pos,
                  float* __restrict__ x, int V, int W, int ldw, int ldx) {
  pdl_enter();
  const int t = blockIdx.x;
  long long id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  const T* src = table + id * ldw;
  const T* add = nullptr;
  if (pos.table) {
    const int p = (pos.pos_dev ? *pos.pos_dev : pos.pos0) + t % pos.S;
    add = static_cast<const T*>(pos.table) + static_cast<long long>(min(max(p, 0), pos.P - 1)) * ldw;
  }
  float* dst = x + static_cast<size_t>(t) * ldx;
  const int whole = (ldw & 7) == 0 ? (W & ~7) : 0;       // columns copied eight at a time
  for (int c = threadIdx.x * 8; c < whole; c += blockDim.x * 8) {
    float f[8];
    load8(src + c, f);
    if (add) {
      float g[8];
      load8(add + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += g[e];
    }
    store8(dst + c, f);
  }
  for (int c = whole + threadIdx.x; c < ldx; c += blockDim.x)
    dst[c] = c < W ? to_f32(src[c]) + (add ? to_f32(add[c]) : 0.f) : 0.f;
}

// out[t, :] = x[t, :] / sqrt(mean(x^2) + eps) * (w + offset), with kCentred of x minus its mean; the
// means run over W columns, rows are ldx apart (a multiple of 8, zero beyond W).  One warp per row.
// NV > 0: the row (at most NV * 256 columns) stays in registers between the reductions and the
// scaling; NV = 0: it is read again for each.
template <typename T, int NV, bool kCentred>
__global__ void __launch_bounds__(128)
rmsnorm_f32_kernel(const float* __restrict__ x, const T* __restrict__ w, float eps, float offset,
                   T* __restrict__ out, int rows, int W, int ldx) {
  pdl_enter();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int lane = threadIdx.x & 31;
  const float* xr = x + static_cast<size_t>(row) * ldx;
  T* orow = out + static_cast<size_t>(row) * ldx;
  constexpr int kBuf = NV ? NV : 1;
  float buf[kBuf][8];
  if constexpr (NV > 0) {
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = (v * 32 + lane) * 8;
      if (c < ldx) load8(xr + c, buf[v]);
    }
  }
  auto each = [&](auto&& fn) {          // fn(column, eight elements) over this lane's columns
    if constexpr (NV > 0) {
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = (v * 32 + lane) * 8;
        if (c < ldx) fn(c, buf[v]);
      }
    } else {
      for (int c = lane * 8; c < ldx; c += 256) {
        load8(xr + c, buf[0]);
        fn(c, buf[0]);
      }
    }
  };
  float mean = 0.f;
  if constexpr (kCentred) {
    float sum = 0.f;
    each([&](int, float (&f)[8]) {
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += f[e];
    });
    mean = warp_add(sum) / static_cast<float>(W);
  }
  float ss = 0.f;
  each([&](int c, float (&f)[8]) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float d = kCentred ? (c + e < W ? f[e] - mean : 0.f) : f[e];
      ss += d * d;
    }
  });
  const float r = 1.0f / sqrtf(warp_add(ss) / static_cast<float>(W) + eps);
  each([&](int c, float (&f)[8]) {
    float wv[8];
    load8(w + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = (f[e] - mean) * r * (wv[e] + offset);
    store8(orow + c, f);
  });
}

// out[m, n] = residual[m, n] + scale * col_scale[n] * act(sum_k a[m, k] b[n, k]), all fp32 (FMA pipe).
// Tile 64 x 64, 256 threads, 4 x 4 outputs per thread.  The order of the additions over k does not
// depend on the number of rows.  With `seg` the grid's third axis is the group: its rows
// [seg[g], seg[g + 1]) of a meet the g-th N rows of b.
constexpr int kTM = 64, kTN = 64, kTK = 16;
__global__ void __launch_bounds__(256)
linear_f32_kernel(const float* __restrict__ a, long long lda, const float* __restrict__ b, const float* residual,
                  const float* __restrict__ col_scale, float scale, int act, float* out,
                  const int* __restrict__ seg, int M, int K, int N) {
  __shared__ float sa[kTK][kTM + 4], sb[kTK][kTN + 4];
  pdl_enter();
  int m0 = blockIdx.y * kTM;
  const int n0 = blockIdx.x * kTN;
  if (seg) {
    m0 += max(seg[blockIdx.z], 0);
    M = min(M, seg[blockIdx.z + 1]);
    b += static_cast<long long>(blockIdx.z) * N * K;
    if (m0 >= M) return;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // this thread's row and k of a tile load
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTK) {
    float4 va = make_float4(0.f, 0.f, 0.f, 0.f), vb = va;
    if (m0 + lr < M && k0 + lk < K) va = *reinterpret_cast<const float4*>(a + (m0 + lr) * lda + k0 + lk);
    if (n0 + lr < N && k0 + lk < K) vb = *reinterpret_cast<const float4*>(b + static_cast<size_t>(n0 + lr) * K + k0 + lk);
    sa[lk][lr] = va.x; sa[lk + 1][lr] = va.y; sa[lk + 2][lr] = va.z; sa[lk + 3][lr] = va.w;
    sb[lk][lr] = vb.x; sb[lk + 1][lr] = vb.y; sb[lk + 2][lr] = vb.z; sb[lk + 3][lr] = vb.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTK; ++k) {
      const float4 fa = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
      const float4 fb = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
      const float av[4] = {fa.x, fa.y, fa.z, fa.w}, bv[4] = {fb.x, fb.y, fb.z, fb.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j];
      if (act == 1) v = fmaxf(v, 0.f) * fmaxf(v, 0.f);
      v *= scale;
      if (col_scale) v *= col_scale[n];
      if (residual) v += residual[static_cast<size_t>(m) * N + n];
      out[static_cast<size_t>(m) * N + n] = v;
    }
  }
}

// h[t, j] = g * sigmoid(alpha g) * (u + offset), g = min(gu[t, j], limit), u = clamp(gu[t, I + j], +-limit)
__global__ void __launch_bounds__(256)
glu_f32_kernel(const float* __restrict__ gu, float* __restrict__ h, long long n, int I, float alpha,
               float limit, float offset) {
  pdl_enter();
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
    const long long t = i / I;
    const int j = static_cast<int>(i - t * I);
    const float g = fminf(gu[t * 2 * I + j], limit);
    const float u = fminf(fmaxf(gu[t * 2 * I + I + j], -limit), limit);
    h[i] = g / (1.0f + expf(-alpha * g)) * (u + offset);
  }
}

template <typename T, bool kCentred>
cudaError_t rmsnorm_any(const float* x, const void* w, float eps, float offset, void* out, int rows, int W,
                        int ldx, cudaStream_t st) {
  auto wp = static_cast<const T*>(w);
  auto op = static_cast<T*>(out);
  const dim3 grid((rows + 3) / 4), block(128);
  const int nv = (ldx + 255) / 256;
#define CDEEP_NORM(NV) return launch_kernel(rmsnorm_f32_kernel<T, NV, kCentred>, grid, block, 0, st, x, wp, eps, offset, op, rows, W, ldx)
  if (nv <= 2) CDEEP_NORM(2);
  if (nv <= 4) CDEEP_NORM(4);
  if (nv <= 8) CDEEP_NORM(8);
  CDEEP_NORM(0);
#undef CDEEP_NORM
}

}  // namespace

cudaError_t launch_embed_rows(const long long* ids, const void* table, float* x, int T, int V, int W, int ldw,
                              int ldx, int fp32, cudaStream_t st, const void* pos, int P, int S, int pos0,
                              const int* pos_dev) {
  if (T == 0) return cudaSuccess;
  const Positions ps{pos, P, S, pos0, pos_dev};
  return fp32 ? launch_kernel(embed_rows_kernel<float>, dim3(T), dim3(128), 0, st, ids,
                              static_cast<const float*>(table), ps, x, V, W, ldw, ldx)
              : launch_kernel(embed_rows_kernel<bf16>, dim3(T), dim3(128), 0, st, ids,
                              static_cast<const bf16*>(table), ps, x, V, W, ldw, ldx);
}

cudaError_t launch_rmsnorm_f32(const float* x, const void* w, float eps, float offset, void* out, int rows, int W,
                               int ldx, int fp32, cudaStream_t st, bool centred) {
  if (rows == 0) return cudaSuccess;
  if (centred)
    return fp32 ? rmsnorm_any<float, true>(x, w, eps, offset, out, rows, W, ldx, st)
                : rmsnorm_any<bf16, true>(x, w, eps, offset, out, rows, W, ldx, st);
  return fp32 ? rmsnorm_any<float, false>(x, w, eps, offset, out, rows, W, ldx, st)
              : rmsnorm_any<bf16, false>(x, w, eps, offset, out, rows, W, ldx, st);
}

cudaError_t launch_linear_f32(const float* a, long long lda, const float* b, const float* residual,
                              const float* col_scale, float scale, int act, float* out, const int* seg, int groups,
                              int M, int K, int N, cudaStream_t st) {
  if (M == 0) return cudaSuccess;
  return launch_kernel(linear_f32_kernel, dim3((N + kTN - 1) / kTN, (M + kTM - 1) / kTM, seg ? groups : 1), dim3(256),
                       0, st, a, lda, b, residual, col_scale, scale, act, out, seg, M, K, N);
}

cudaError_t launch_glu_f32(const float* gu, float* h, int T, int I, float alpha, float limit, float offset,
                           cudaStream_t st) {
  const long long n = static_cast<long long>(T) * I;
  if (n == 0) return cudaSuccess;
  const long long blocks = (n + 255) / 256;
  return launch_kernel(glu_f32_kernel, dim3(static_cast<unsigned>(blocks < 4096 ? blocks : 4096)), dim3(256), 0, st, gu,
                       h, n, I, alpha, limit, offset);
}

}  // namespace cdeep

// Shared description of attention over a sliding window with kept first tokens, a per-head
// distance bias and mixing of the heads' weights.
//
//   s_h(i, j) = scale q_h(i) . k_c(j) - r1_h ln(1 + r2_h (i - j)),  c = h / (H / G)
//   w_h(i, .) = softmax over { j <= i : i - j < window or j < keep }
//   o_h(i)    = sum_j (sum_g talk[h, g] w_g(i, j)) v_c(j)
//
// Keys and values of earlier calls live in a ring of keep + window slots per sequence: position
// j < keep has slot j for good, any other position slot keep + (j - keep) % window.  The slot of
// position i therefore held position i - window, which position i does not see.
#pragma once
#include "../../include/cdeep.h"
#include "elem.cuh"

namespace cdeep {

using WindowAttnParams = cd_window_attn;

__device__ __forceinline__ int window_slot(int j, int window, int keep) {
  return j < keep ? j : keep + (j - keep) % window;
}
__device__ __forceinline__ int window_pos0(const WindowAttnParams& p) { return p.pos_dev ? __ldg(p.pos_dev) : p.pos0; }

// Keys of query i as one run of indices n = 0 .. count - 1: first the kept tokens that the window
// does not reach, then the window.
struct WindowKeys {
  int kept;    // kept tokens before the window
  int first;   // first position of the window
  __device__ __forceinline__ WindowKeys(int lo_query, int window, int keep) {
    first = lo_query - window + 1;
    if (first < 0) first = 0;
    kept = keep < first ? keep : first;
  }
  __device__ __forceinline__ int position(int n) const { return n < kept ? n : first + (n - kept); }
};

}  // namespace cdeep

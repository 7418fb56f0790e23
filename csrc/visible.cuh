// Which keys a causal query sees besides "no later ones": a sliding window, or fixed chunks of the sequence.
#pragma once

namespace icb {

struct Visible {
  int window;      // the `window` tokens that end with the query itself (0: no limit)
  int chunk;       // keys of the query's own chunk of `chunk` tokens, counted from the sequence's start (0: no limit)
};

// First position that a query at `pos` sees.
__device__ __forceinline__ int first_visible(const Visible& v, int pos) {
  int lo = 0;
  if (v.window > 0) lo = max(lo, pos - v.window + 1);
  if (v.chunk > 0) lo = max(lo, pos / v.chunk * v.chunk);
  return lo;
}

}  // namespace icb

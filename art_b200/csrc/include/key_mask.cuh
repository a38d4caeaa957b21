// Which keys a position sees besides being causal: the last `window` ones (itself included), or those of its own chunk of
// the sequence, chunks counted from position 0.  0 switches either off.
#pragma once

namespace artb {

struct KeyMask {
  int window, chunk;
  // first key position p sees
  __host__ __device__ __forceinline__ int first(int p) const {
    int lo = window > 0 && p >= window ? p - window + 1 : 0;
    if (chunk > 0) {
      const int c = p - p % chunk;
      if (c > lo) lo = c;
    }
    return lo;
  }
};

}  // namespace artb

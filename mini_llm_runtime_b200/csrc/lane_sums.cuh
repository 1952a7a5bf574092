// Sums of several values at once over groups of lanes.
#pragma once

#include "common.cuh"

namespace mlr {

// N values per lane summed over groups of SL lanes (SL a power of two): halves of the values are exchanged
// until a lane holds one value (then plain sums), so that the N totals end up spread over the group.
// Returns the index of the lane's first total; it holds max(1, N / SL) of them, in v[0 ..].
template <int N, int SL>
__device__ __forceinline__ int spread_sums(float (&v)[N], int lane) {
  int index = 0, live = N;
#pragma unroll
  for (int m = SL / 2; m > 0; m >>= 1) {
    if (live > 1) {
      const bool upper = (lane & m) != 0;
      live >>= 1;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < live) {
          const float send = upper ? v[i] : v[i + live];
          const float keep = upper ? v[i + live] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
      }
      if (upper) index += live;
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
    }
  }
  return index;
}

}  // namespace mlr

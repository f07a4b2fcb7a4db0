// Work items of a ragged step: the rows of every segment cut into pieces of at most `piece` rows.
#pragma once

#include "common.cuh"

namespace cb200 {

struct RaggedItem {
  int seg;      // -1: no such item
  int row0;     // first row of the item
  int count;    // its rows
  int first;    // index of the segment's first item
  bool last;    // the segment's last item
};

// Item `index` in segment order, found by one warp (every lane gets the result). cu_rows has segments + 1 entries.
__device__ __forceinline__ RaggedItem find_item(const int32_t* __restrict__ cu_rows, int segments, int piece, int index) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int base = 0; base < segments; base += 32) {
    const int s = base + lane;
    const int n = s < segments ? cu_rows[s + 1] - cu_rows[s] : 0;
    const int items = (n + piece - 1) / piece;
    int incl = items;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, incl, off);
      if (lane >= off) incl += up;
    }
    const int start = before + incl - items;
    const unsigned hit = __ballot_sync(0xffffffffu, index >= start && index < start + items);
    if (hit != 0u) {
      const int src = __ffs(hit) - 1;
      RaggedItem it;
      it.seg = base + src;
      it.first = __shfl_sync(0xffffffffu, start, src);
      const int rows = __shfl_sync(0xffffffffu, n, src);
      const int k = index - it.first;
      it.row0 = cu_rows[it.seg] + k * piece;
      it.count = min(piece, rows - k * piece);
      it.last = (k + 1) * piece >= rows;
      return it;
    }
    before += __shfl_sync(0xffffffffu, incl, 31);
  }
  return RaggedItem{-1, 0, 0, 0, false};
}

// Upper bound of the item count of any step with these extents.
inline int ragged_items(int rows, int segments, int piece) { return rows / piece + segments; }

}  // namespace cb200

// Segments of a batch (runs of consecutive positions of one slot) for kernels that walk them row by row: from a host table (first row, row
// count), or without one from the slots of the rows themselves, where the first row of a slot takes all rows of it. A: has slot, seg_first,
// seg_count (null: no table) and rows.
#pragma once
#include "common.cuh"

namespace ve {

// First row of the segment that z stands for (z counts segments of the table, or rows); -1 when there is nothing to do. count: its rows (-1:
// they are found while walking).
template <typename A>
VE_DEVINL int segment_of(const A& a, int z, int& count) {
  if (a.seg_first) {
    count = a.seg_count[z];
    return count > 0 ? a.seg_first[z] : -1;
  }
  const int s = a.slot[z];
  if (s < 0) return -1;
  for (int i = 0; i < z; ++i)
    if (a.slot[i] == s) return -1;
  count = -1;
  return z;
}
template <typename A>
VE_DEVINL int next_row(const A& a, int i, int left) {
  if (a.seg_first) return left > 1 ? i + 1 : -1;
  const int s = a.slot[i];
  for (int j = i + 1; j < a.rows; ++j)
    if (a.slot[j] == s) return j;
  return -1;
}

}  // namespace ve

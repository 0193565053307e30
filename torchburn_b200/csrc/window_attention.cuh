// The positions a row sees under a sliding window with kept first positions.
#pragma once

namespace tb {

struct VisibleRange {
  int nk = 0;    // visible positions in front of the window (0..nk-1)
  int lo = 0;    // first position of the window's run
  int hi = -1;   // the row's own position
  __host__ __device__ VisibleRange(int pos, int window, int keep_first) {
    hi = pos;
    lo = pos - window + 1 > 0 ? pos - window + 1 : 0;
    nk = keep_first < lo ? keep_first : lo;   // kept positions inside the window belong to its run
  }
  __host__ __device__ int count() const { return hi < 0 ? 0 : nk + hi - lo + 1; }
  __host__ __device__ int position(int v) const { return v < nk ? v : v - nk + lo; }
};

}  // namespace tb

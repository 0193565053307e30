// The positions a row sees under a sliding window with kept first positions, or inside its chunk of the sequence,
// and how the keys of a block of rows are numbered.
#pragma once

#include "dense.cuh"

namespace tb {

struct VisibleRange {
  int nk = 0;    // visible positions in front of the window (0..nk-1)
  int lo = 0;    // first position of the window's run
  int hi = -1;   // the row's own position
  // chunk > 0: the run also begins at the row's own chunk, chunks counted from position 0
  __host__ __device__ VisibleRange(int pos, int window, int keep_first, int chunk = 0) {
    hi = pos;
    lo = pos - window + 1 > 0 ? pos - window + 1 : 0;
    if (chunk > 0 && pos >= 0) {
      const int start = pos - pos % chunk;
      lo = start > lo ? start : lo;
    }
    nk = keep_first < lo ? keep_first : lo;   // kept positions inside the window belong to its run
  }
  __host__ __device__ int count() const { return hi < 0 ? 0 : nk + hi - lo + 1; }
  __host__ __device__ int position(int v) const { return v < nk ? v : v - nk + lo; }
};

// The keys of a block of consecutive rows: the kept positions, then one run from the first row's window to the last
// row.  p0: position of the block's first row, last: of its last one.
struct BlockKeys {
  int pos0, lo, nk, count;
  __host__ __device__ BlockKeys(int p0, int last, int window, int keep_first, int chunk = 0) : pos0(p0) {
    const VisibleRange a(p0, window, keep_first, chunk);
    lo = a.lo;
    nk = a.nk;
    count = last < 0 ? 0 : nk + last - lo + 1;
  }
  __host__ __device__ int position(int v) const { return v < nk ? v : v - nk + lo; }
};

// Cache rows of numbered keys near number v0 (less than a ring apart) with one division for all of them.
struct RunRows {
  int nk, lo, keep, ring, base_pos, base_row;
  __host__ __device__ RunRows(const BlockKeys& k, const CacheGeom& g, int v0) : nk(k.nk), lo(k.lo), keep(g.keep), ring(g.ring) {
    const int p = k.position(v0 > k.nk ? v0 : k.nk);   // first key of the run at or after v0
    base_pos = p > keep ? p : keep;
    base_row = g.row_of(base_pos);
  }
  __host__ __device__ int row(int v) const {
    const int p = v < nk ? v : v - nk + lo;
    if (ring == 0 || p < keep) return p;
    const int r = base_row + (p - base_pos);
    return r >= keep + ring ? r - ring : r;
  }
};

}  // namespace tb

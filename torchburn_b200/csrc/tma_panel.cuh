// Panels of 64 bf16 columns of a row-major matrix by TMA, with the tensor core's 128-byte swizzle on the way.
#pragma once

#include <climits>

#include <cuda.h>

#include "dense.cuh"

namespace tb {

#ifdef __CUDACC__
// The panel from column x, row y on; x on a 16-byte boundary.  Columns and rows outside the matrix are zeros.
__device__ __forceinline__ void tma_panel(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst), "l"(map), "r"(x),
               "r"(y), "r"(bar)
               : "memory");
}
#endif

// Panels of `panel_rows` rows; false when the matrix cannot be described (alignment, sizes) or the driver lacks the call.
inline bool tma_panel_map(CUtensorMap* map, const void* base, int64_t cols, int64_t rows, int64_t stride, int panel_rows) {
  using Encode = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                              const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
  static const Encode encode = [] {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult found;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &fn, 12000, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess) fn = nullptr;
    return reinterpret_cast<Encode>(fn);
  }();
  if (!encode || rows < 1 || rows > INT_MAX) return false;
  const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)stride * 2};
  const cuuint32_t box[2] = {64, (cuuint32_t)panel_rows}, steps[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, steps, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace tb

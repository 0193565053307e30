// What the kernels of flash_attention.cu and flash_tc5.cu share.
#pragma once

#include "dense.cuh"

namespace tb {

struct FlashShape {
  int run_rows = 0;   // rows that share a sequence: the whole step, or one
  int tiles = 0;      // CTAs' shares of a run's (query, head) pairs
  int splits = 1;     // CTAs that share a tile's keys
};

// Elements behind a head's output that the next product's padded K covers: column c of head h for c in [vdim, limit).
__host__ __device__ __forceinline__ int flash_column_limit(const FlashArgs& a, int h) {
  if (a.out_per_head) return a.out.kp;
  return h == a.heads - 1 ? a.out.kp - h * a.vdim : a.vdim;
}

#ifdef __CUDACC__
template <bool BF16>
__device__ __forceinline__ void flash_store_column(const FlashArgs& a, int row, int h, int c, float v) {
  if (!a.out_per_head) {
    act_store1<BF16>(a.out, row, h * a.vdim + c, v);
    return;
  }
  ActOperand o = a.out;
  o.data = static_cast<unsigned char*>(o.data) + (size_t)h * o.mp * o.kp * (BF16 ? 2 : 4);
  act_store1<BF16>(o, row, c, v);
}
#endif

// Decode steps over latents on tcgen05 (flash_latent.cu); leaves parts for a merge when *splits > 1.
bool flash_latent_supported(const FlashArgs& a);
tb_status launch_flash_latent(const FlashArgs& a, cudaStream_t st, int* splits);

// Portions of one sequence on tcgen05 (flash_tc5.cu); leaves parts for a merge when *splits > 1.
bool flash_tc5_supported(const FlashArgs& a);
tb_status launch_flash_tc5(const FlashArgs& a, cudaStream_t st, int* splits);

}  // namespace tb

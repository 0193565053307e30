// Unquantized projections y = W x of the layered decoder.
//
// bf16: tcgen05.  The weights are the M = 128 side of the MMA (a CTA owns 128 output features), the
// activation rows its N = 16..256.  Both operands lie in global memory as ready-made 128-byte-swizzled
// K-major images (dense.cuh), so a pipeline stage is two bulk copies; one thread issues the MMAs, four
// warps read the fp32 accumulator back (thread = output feature, so a store is 32 consecutive floats).
// From one decode row to a whole prompt portion it is the same kernel: with few rows it streams the
// weights (several CTAs per SM, K split over CTAs when there are fewer tiles than SMs), with many rows it
// is bound by the tensor core.  A K split writes partial sums which the consuming row kernel adds in a
// fixed order; without one the epilogue can also write the next kernel's input itself (rows of the activation
// type, or an activated operand image).  A batch of matrices (one per head) is one launch.  The weight copies of the first stages are issued before the grid dependency wait: weights
// depend on nothing, so with programmatic launch they overlap the previous kernel's tail.
//
// fp32: a shared-memory tiled product on the CUDA cores, every product and sum in fp32.
#include "dense.cuh"
#include "tc5.cuh"

namespace tb {

namespace {

using namespace tc5;

constexpr int kTile = 128;            // output features per CTA
constexpr int kTileBytes = 16384;     // 128 rows x 64 bf16
constexpr int kShortLoop = 16;        // K blocks

__device__ int g_dense_fault = 0;

struct GemmParams {
  const unsigned char* w;
  const unsigned char* x;
  void* out;
  int64_t ldo, n_valid, batch_cols;
  size_t split_stride, w_batch, x_batch;
  ActOperand operand;
  DenseSink sink;
  DenseAct act;
  int rows, mp, kb, kb_per, splits;
};

__device__ __forceinline__ float activate(DenseAct act, float v) {
  if (act == DenseAct::kRelu2) {
    v = fmaxf(v, 0.f);
    return v * v;
  }
  return v;
}
// One sum that is not partial.
template <bool BF16>
__device__ __forceinline__ void store_sum(const GemmParams& p, int row, int64_t col, float v) {
  v = activate(p.act, v);
  if (p.sink == DenseSink::kOperand) act_store1<BF16>(p.operand, row, (int)col, v);
  else if (BF16) static_cast<__nv_bfloat16*>(p.out)[(size_t)row * p.ldo + col] = __float2bfloat16_rn(v);
  else static_cast<float*>(p.out)[(size_t)row * p.ldo + col] = v;
}

template <int BN, int STAGES>
__global__ void __launch_bounds__(192) dense_tc5_kernel(const GemmParams p) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES], done;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  constexpr int kBBytes = BN * 128, kStage = kTileBytes + kBBytes;
  constexpr int kCols = BN < 32 ? 32 : BN;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int row0 = (int)blockIdx.x * BN;
  const int split = (int)blockIdx.z % p.splits, batch = (int)blockIdx.z / p.splits;
  const int kb0 = split * p.kb_per;
  const int nkb = min(p.kb - kb0, p.kb_per);

  if (tid == 0) {
    s_abort = 0;
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(kCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  grid_dep_launch();
  const uint32_t tmem = s_tmem;

  if (warp == 4) {
    if (lane == 0) {   // ---- copies ----
      const unsigned char* wsrc = p.w + (size_t)batch * p.w_batch + ((size_t)blockIdx.y * p.kb + kb0) * kTileBytes;
      const unsigned char* xsrc = p.x + (size_t)batch * p.x_batch + (size_t)kb0 * ((size_t)p.mp * 128) + (size_t)row0 * 128;
      const int pre = nkb < STAGES ? nkb : STAGES;
      for (int i = 0; i < pre; ++i) {
        mbar_expect_tx(&full[i], kStage);
        bulk_g2s(smem + (size_t)i * kStage, wsrc + (size_t)i * kTileBytes, kTileBytes, &full[i]);
      }
      grid_dep_wait();
      for (int i = 0; i < pre; ++i)
        bulk_g2s(smem + (size_t)i * kStage + kTileBytes, xsrc + (size_t)i * ((size_t)p.mp * 128), kBBytes, &full[i]);
      int issued = pre;
      for (int i = pre; i < nkb; ++i) {
        const int s = i % STAGES;
        if (!mbar_wait(&empty[s], (uint32_t)(i / STAGES - 1) & 1u, &s_abort, &g_dense_fault)) break;
        mbar_expect_tx(&full[s], kStage);
        bulk_g2s(smem + (size_t)s * kStage, wsrc + (size_t)i * kTileBytes, kTileBytes, &full[s]);
        bulk_g2s(smem + (size_t)s * kStage + kTileBytes, xsrc + (size_t)i * ((size_t)p.mp * 128), kBBytes, &full[s]);
        issued = i + 1;
      }
      // copies in flight must have landed before the CTA gives its shared memory back
      for (int i = issued > STAGES ? issued - STAGES : 0; i < issued; ++i) {
        int no_abort = 0;
        mbar_wait(&full[i % STAGES], (uint32_t)(i / STAGES) & 1u, &no_abort, &g_dense_fault);
      }
    }
  } else if (warp == 5) {
    if (lane == 0) {   // ---- MMA issue ----
      // fp32 accumulator, bf16 x bf16, both K-major, N = BN, M = 128
      constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kTile >> 4) << 24);
      for (int i = 0; i < nkb; ++i) {
        const int s = i % STAGES;
        if (!mbar_wait(&full[s], (uint32_t)(i / STAGES) & 1u, &s_abort, &g_dense_fault)) break;
        tc_fence_after();
        const uint32_t a_lo = (smem_u32(smem + (size_t)s * kStage) >> 4) | (1u << 16);
        const uint32_t b_lo = (smem_u32(smem + (size_t)s * kStage + kTileBytes) >> 4) | (1u << 16);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)   // 16 bf16 = 32 bytes of a row per MMA
          mma_bf16_ss(tmem, a_lo + (uint32_t)(ks * 2), b_lo + (uint32_t)(ks * 2), idesc, (i | ks) != 0 ? 1u : 0u);
        mma_commit(&empty[s]);
      }
      mma_commit(&done);
      int no_abort = 0;
      mbar_wait(&done, 0u, &no_abort, &g_dense_fault);
    }
  } else {
    // ---- epilogue: thread = output feature, columns of tensor memory = activation rows ----
    bool ok = true;
    if (lane == 0) ok = mbar_wait(&done, 0u, &s_abort, &g_dense_fault);
    __syncwarp();
    ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
    if (ok) {
      tc_fence_after();
      const int64_t n = (int64_t)blockIdx.y * kTile + warp * 32 + lane;
      const bool live = n < p.n_valid;
      const uint32_t base = tmem + ((uint32_t)(warp * 32) << 16);
      float* dst = static_cast<float*>(p.out) + (size_t)split * p.split_stride + (size_t)row0 * p.ldo + n;
      const int64_t col = (int64_t)batch * p.batch_cols + n;
      const int nrows = min(p.rows - row0, BN);
      // eight features of a row lie side by side, on a 16-byte boundary
      const bool wide = p.sink != DenseSink::kPartials && ((p.n_valid | p.batch_cols | (p.sink == DenseSink::kRows ? p.ldo : 0)) & 7) == 0;
#pragma unroll 1
      for (int c = 0; c < nrows; c += 16) {
        uint32_t r[2][8];
        tmem_ld8(base + (uint32_t)c, r[0]);
        tmem_ld8(base + (uint32_t)c + 8, r[1]);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (live && p.sink == DenseSink::kPartials) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c + j < nrows) dst[(size_t)(c + j) * p.ldo] = __uint_as_float(r[j >> 3][j & 7]);
        } else if (wide) {
          // through the warp's corner of the first stage (every MMA has read it): 16 rows x 32 features, then 8 features
          // per store
          __nv_bfloat16* t = reinterpret_cast<__nv_bfloat16*>(smem) + warp * (16 * 40);
#pragma unroll
          for (int j = 0; j < 16; ++j) t[j * 40 + lane] = __float2bfloat16_rn(activate(p.act, __uint_as_float(r[j >> 3][j & 7])));
          __syncwarp();
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int j = (lane >> 2) + h * 8, f = (lane & 3) * 8;
            if (c + j < nrows && n - lane + f < p.n_valid) {
              const uint4 v = *reinterpret_cast<const uint4*>(t + j * 40 + f);
              const int64_t k = col - lane + f;
              if (p.sink == DenseSink::kOperand)
                *reinterpret_cast<uint4*>(static_cast<unsigned char*>(p.operand.data) + image_offset(p.operand.mp, row0 + c + j, (int)k)) = v;
              else *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + (size_t)(row0 + c + j) * p.ldo + k) = v;
            }
          }
          __syncwarp();
        } else if (live) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c + j < nrows) store_sum<true>(p, row0 + c + j, col, __uint_as_float(r[j >> 3][j & 7]));
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kCols) : "memory");
  }
}

// RPT rows per thread: a CTA covers 128 output features x 8 * RPT activation rows.
template <int RPT>
__global__ void __launch_bounds__(256) dense_f32_kernel(const GemmParams p) {
  constexpr int ROWS = 8 * RPT;
  __shared__ float ws[64][kTile];
  __shared__ float xs[ROWS][64];
  const int tid = threadIdx.x;
  const int row0 = (int)blockIdx.x * ROWS;
  const int kp = p.kb * 64;
  const int split = (int)blockIdx.z % p.splits, batch = (int)blockIdx.z / p.splits;
  const float* x = reinterpret_cast<const float*>(p.x + (size_t)batch * p.x_batch);
  grid_dep_launch();
  grid_dep_wait();
  const int n4 = (tid & 31) * 4, rg = tid >> 5;   // 4 features, rows rg + 8 i
  float acc[RPT][4];
#pragma unroll
  for (int i = 0; i < RPT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const int kb0 = split * p.kb_per, kb1 = min(p.kb, kb0 + p.kb_per);
  for (int kb = kb0; kb < kb1; ++kb) {
    const unsigned char* tile = p.w + (size_t)batch * p.w_batch + ((size_t)blockIdx.y * p.kb + kb) * kTileBytes;
    for (int c = tid; c < kTile * 8; c += 256) {    // 16-byte pieces: feature c & 127, piece c >> 7
      const int n = c & 127, pc = c >> 7;
      const uint4 v = *reinterpret_cast<const uint4*>(tile + n * 128 + ((pc ^ (n & 7)) << 4));
      const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        ws[pc * 8 + 2 * j][n] = __uint_as_float(u[j] << 16);
        ws[pc * 8 + 2 * j + 1][n] = __uint_as_float(u[j] & 0xFFFF0000u);
      }
    }
    for (int i = tid; i < ROWS * 64; i += 256) {
      const int r = i >> 6, k = i & 63;
      xs[r][k] = row0 + r < p.rows ? x[(size_t)(row0 + r) * kp + kb * 64 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < 64; ++k) {
      const float4 w = *reinterpret_cast<const float4*>(&ws[k][n4]);
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const float v = xs[rg + 8 * i][k];
        acc[i][0] = fmaf(v, w.x, acc[i][0]);
        acc[i][1] = fmaf(v, w.y, acc[i][1]);
        acc[i][2] = fmaf(v, w.z, acc[i][2]);
        acc[i][3] = fmaf(v, w.w, acc[i][3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int row = row0 + rg + 8 * i;
    if (row >= p.rows) continue;
    float* dst = static_cast<float*>(p.out) + (size_t)split * p.split_stride + (size_t)row * p.ldo;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t n = (int64_t)blockIdx.y * kTile + n4 + j;
      if (n >= p.n_valid) continue;
      if (p.sink == DenseSink::kPartials) dst[n] = acc[i][j];
      else store_sum<false>(p, row, (int64_t)batch * p.batch_cols + n, acc[i][j]);
    }
  }
}

// bf16 [batch][n, k], element (r, c) of a matrix at r * sn + c * sk -> tile images (rows row0..row0+n of each matrix).
__global__ void __launch_bounds__(256) pack_weight_kernel(const uint16_t* __restrict__ src, unsigned char* __restrict__ img, int64_t row0,
                                                          int64_t n, int64_t k, int64_t kp, int64_t sn, int64_t sk, int64_t img_batch, int batch) {
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;   // one 16-byte piece
  const int64_t pieces = kp >> 3;
  if (i >= batch * n * pieces) return;
  const int64_t rb = i / pieces, pc = i - rb * pieces, b = rb / n, r = rb - b * n;
  src += b * n * k;
  img += b * img_batch;
  uint16_t v[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int64_t kk = pc * 8 + j;
    v[j] = kk < k ? src[r * sn + kk * sk] : (uint16_t)0;
  }
  const int64_t row = row0 + r, kb = pc >> 3;
  unsigned char* dst = img + ((row >> 7) * (kp >> 6) + kb) * kTileBytes + (row & 127) * 128 + (((pc & 7) ^ (row & 7)) << 4);
  uint4 u;
  u.x = v[0] | ((uint32_t)v[1] << 16); u.y = v[2] | ((uint32_t)v[3] << 16);
  u.z = v[4] | ((uint32_t)v[5] << 16); u.w = v[6] | ((uint32_t)v[7] << 16);
  *reinterpret_cast<uint4*>(dst) = u;
}

template <int BN, int STAGES>
tb_status launch_tc5(const GemmParams& p, int n_tiles, unsigned nz, bool pdl, cudaStream_t st) {
  const size_t smem = (size_t)STAGES * (kTileBytes + BN * 128) + 1024;
  return launch_kernel(dense_tc5_kernel<BN, STAGES>, dim3((unsigned)((p.rows + BN - 1) / BN), (unsigned)n_tiles, nz), dim3(192),
                       smem, st, pdl, 1, p);
}

}  // namespace

int dense_fault_flag() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_dense_fault, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

tb_status dense_weight_alloc(DenseWeight* w, int64_t rows, int64_t k, int batch) {
  w->rows = pad_to(rows, kTile);
  w->kp = pad_to(k, kPad);
  w->batch = batch;
  const size_t bytes = (size_t)w->rows * w->kp * 2 * (size_t)batch;
  TB_CUDA_TRY(cudaMalloc(&w->img, bytes));
  TB_CUDA_TRY(cudaMemset(w->img, 0, bytes));
  return TB_OK;
}

tb_status dense_weight_fill(DenseWeight* w, int64_t row0, const uint16_t* src, int64_t n, int64_t k, tb_space space, bool transposed) {
  if (!src) return fail(TB_ERR_ARG, "dense weight: null tensor");
  void* tmp = nullptr;
  if (space == TB_HOST) TB_TRY(upload(&tmp, src, (size_t)w->batch * n * k * 2, TB_HOST));
  const int64_t pieces = w->batch * n * (w->kp >> 3);
  pack_weight_kernel<<<(unsigned)((pieces + 255) / 256), 256>>>(space == TB_HOST ? static_cast<const uint16_t*>(tmp) : src,
                                                               static_cast<unsigned char*>(w->img), row0, n, k, w->kp, transposed ? 1 : k,
                                                               transposed ? n : 1, w->rows * w->kp * 2, w->batch);
  const cudaError_t e = cudaGetLastError();
  const cudaError_t e2 = cudaDeviceSynchronize();
  cudaFree(tmp);
  TB_CUDA_TRY(e);
  TB_CUDA_TRY(e2);
  return TB_OK;
}

int dense_row_pad(int rows) {
  if (rows <= 16) return 16;
  if (rows <= 32) return 32;
  if (rows <= 64) return 64;
  return (int)pad_to(rows, rows <= 128 ? 128 : 256);
}

int dense_splits(Precision p, int64_t n_rows, int64_t kp, int rows, int max_splits, double* gain) {
  if (gain) *gain = 0.0;
  if (p == Precision::kF32) return 1;
  const int mp = dense_row_pad(rows);
  const int tiles = (int)(n_rows / kTile) * (mp > 256 ? mp / 256 : 1);
  const int kb = (int)(kp / 64);
  // CTAs that fit side by side: two per SM with few rows, one with wide row tiles
  const int slots = sm_count() * (mp <= 64 ? 2 : 1);
  int best = 1;
  double best_cost = 1e30, whole = 0.0;
  for (int s = 1; s <= max_splits && s <= kb; ++s) {
    const int per = (kb + s - 1) / s;
    if ((kb + per - 1) / per != s) continue;   // no empty split
    const double waves = (double)((tiles * s + slots - 1) / slots);
    const double cost = waves * (per + 6.0) + 0.5 * s;   // 6: fixed cost of a CTA in stages; partial sums cost the consumer
    if (s == 1) whole = cost;
    if (cost < best_cost - 1e-9) { best_cost = cost; best = s; }
  }
  if (gain) *gain = whole - best_cost;
  return best;
}

tb_status launch_dense_gemm(Precision prec, const DenseGemmArgs& a, cudaStream_t st) {
  if (a.rows < 1 || a.x.kp != a.w->kp) return fail(TB_ERR_SHAPE, "dense product: rows %d, K %d against %lld", a.rows, a.x.kp, (long long)a.w->kp);
  GemmParams p;
  p.w = static_cast<const unsigned char*>(a.w->img);
  p.x = static_cast<const unsigned char*>(a.x.data);
  p.out = a.out; p.ldo = a.ldo; p.n_valid = a.n_valid; p.split_stride = a.split_stride; p.batch_cols = a.batch_cols;
  p.operand = a.operand; p.sink = a.sink; p.act = a.act; p.splits = a.splits;
  p.w_batch = (size_t)a.w->rows * a.w->kp * 2;
  p.x_batch = (size_t)a.x.mp * a.x.kp * (prec == Precision::kBf16 ? 2 : 4);
  if (a.splits != 1 && a.sink != DenseSink::kPartials) return fail(TB_ERR_SHAPE, "dense product: %d partial sums cannot be activated", a.splits);
  const unsigned nz = (unsigned)(a.splits * a.w->batch);
  p.rows = a.rows; p.mp = a.x.mp; p.kb = (int)(a.w->kp / 64);
  p.kb_per = (p.kb + a.splits - 1) / a.splits;
  if ((p.kb + p.kb_per - 1) / p.kb_per != a.splits) return fail(TB_ERR_SHAPE, "dense product: %d splits of %d K blocks", a.splits, p.kb);
  const int n_tiles = (int)(a.w->rows / kTile);
  if (prec == Precision::kF32) {
    if (a.rows > 8)
      return launch_kernel(dense_f32_kernel<8>, dim3((unsigned)((a.rows + 63) / 64), (unsigned)n_tiles, nz), dim3(256), 0, st, a.pdl, 1, p);
    return launch_kernel(dense_f32_kernel<1>, dim3(1, (unsigned)n_tiles, nz), dim3(256), 0, st, a.pdl, 1, p);
  }
  if (a.x.mp != dense_row_pad(a.rows)) return fail(TB_ERR_SHAPE, "dense product: operand padded to %d rows for %d", a.x.mp, a.rows);
  switch (p.mp) {
    case 16: return launch_tc5<16, 6>(p, n_tiles, nz, a.pdl, st);
    case 32: return launch_tc5<32, 5>(p, n_tiles, nz, a.pdl, st);
    case 64: return launch_tc5<64, 4>(p, n_tiles, nz, a.pdl, st);
    case 128: return launch_tc5<128, 6>(p, n_tiles, nz, a.pdl, st);
    default:
      // a short K loop is mostly epilogue: two CTAs per SM, one stores while the other computes
      if (p.kb_per <= kShortLoop && (int64_t)(p.mp / 256) * n_tiles * nz > sm_count()) return launch_tc5<256, 2>(p, n_tiles, nz, a.pdl, st);
      return launch_tc5<256, 4>(p, n_tiles, nz, a.pdl, st);
  }
}

}  // namespace tb

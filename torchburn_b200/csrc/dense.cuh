// Kernels of the layered decoder (layered.cu): unquantized projections, the row kernels between them, flash
// attention and windowed attention with mixed heads.  Everything is a parameter: sizes, windows, taps, constants.
//
// Precision.  With 16-bit products (Precision::kBf16) the operands of a projection are bf16 and the sums
// fp32; the residual stream, norms, scores, attention weights and the convolution history are fp32, the KV
// cache bf16.  With Precision::kF32 activations, caches and every product are fp32 (weights are stored as
// bf16 either way: the checkpoints hold bf16 values, which fp32 represents exactly).
//
// Padding.  The feature dimension of every vector is padded with zeros to a multiple of 64 (kPad), the
// output rows of a weight matrix to a multiple of 128; padded weights are zero, so padded outputs are zero.
#pragma once

#include <cuda_bf16.h>

#include "tb_common.cuh"

namespace tb {

enum class Precision { kBf16 = 0, kF32 = 1 };

constexpr int64_t kPad = 64;
inline int64_t pad_to(int64_t v, int64_t m) { return (v + m - 1) / m * m; }

// ---- operand of a projection -------------------------------------------------------------------
// bf16: per 64 elements of K one image of [mp rows x 128 bytes], the 16-byte pieces of a row XORed with
// the row number (the 128-byte swizzle of the tensor core's shared-memory tiles), so that a tile is one
// contiguous bulk copy.  fp32: row-major [mp, kp].
struct ActOperand {
  void* data = nullptr;
  int mp = 0;   // padded rows
  int kp = 0;   // padded K
};
#ifdef __CUDACC__
__device__ __forceinline__ size_t image_offset(int mp, int row, int k) {   // bytes
  return (size_t)(k >> 6) * ((size_t)mp * 128) + (size_t)row * 128 + (size_t)((((k >> 3) & 7) ^ (row & 7)) << 4) + (size_t)((k & 7) << 1);
}
template <bool BF16>
__device__ __forceinline__ void act_store1(const ActOperand& a, int row, int k, float v) {
  if (BF16) *reinterpret_cast<__nv_bfloat16*>(static_cast<unsigned char*>(a.data) + image_offset(a.mp, row, k)) = __float2bfloat16_rn(v);
  else static_cast<float*>(a.data)[(size_t)row * a.kp + k] = v;
}
// four consecutive elements, k a multiple of 4
template <bool BF16>
__device__ __forceinline__ void act_store4(const ActOperand& a, int row, int k, float4 v) {
  if (BF16) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    *reinterpret_cast<uint2*>(static_cast<unsigned char*>(a.data) + image_offset(a.mp, row, k)) = u;
  } else {
    *reinterpret_cast<float4*>(static_cast<float*>(a.data) + (size_t)row * a.kp + k) = v;
  }
}
__device__ __forceinline__ void grid_dep_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void grid_dep_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
#endif

// Launch with optional programmatic stream serialization and a cluster of `cluster` CTAs along x.
template <typename... KArgs, typename... Args>
tb_status launch_kernel(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl, int cluster, Args... args) {
  if (smem > 48 * 1024) TB_CUDA_TRY(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (cluster > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = (unsigned)cluster;
    attr[n].val.clusterDim.y = 1;
    attr[n++].val.clusterDim.z = 1;
  }
  cfg.attrs = attr;
  cfg.numAttrs = (unsigned)n;
  TB_CUDA_TRY(cudaLaunchKernelEx(&cfg, kern, args...));
  return TB_OK;
}

// ---- projections (dense_gemm.cu) ---------------------------------------------------------------
// A weight matrix [n, k] as tiles of 128 rows x 64 columns, each a contiguous 16 KB image like
// ActOperand's: tile (n / 128, k / 64) at ((n / 128) * (kp / 64) + k / 64) * 16384 bytes.  `batch` matrices of
// one size (one per head, say) lie one after the other.
struct DenseWeight {
  void* img = nullptr;
  int64_t rows = 0;   // padded rows (multiple of 128)
  int64_t kp = 0;     // padded K (multiple of 64)
  int batch = 1;
};
tb_status dense_weight_alloc(DenseWeight* w, int64_t rows, int64_t k, int batch = 1);
// Rows [row0, row0 + n) of every matrix of the batch from bf16 matrices [batch][n, k] (host or device);
// `transposed`: each is stored as [k, n].
tb_status dense_weight_fill(DenseWeight* w, int64_t row0, const uint16_t* src, int64_t n, int64_t k, tb_space space, bool transposed = false);

// Partial sums of a projection: y[s][row][ldy], s < splits <= 8; the consumer adds them in that order.
struct PartialSums {
  float* y = nullptr;
  int splits = 1;
  size_t split_stride = 0;   // floats
  int64_t ldy = 0;
};
// Where a product's sums go: fp32 partial sums for a row kernel, rows of the activation type (bf16 or fp32), or,
// after an elementwise activation, the operand of the next product.
enum class DenseSink { kPartials = 0, kRows = 1, kOperand = 2 };
enum class DenseAct { kNone = 0, kRelu2 = 1 };   // kRelu2: the square of max(z, 0)
struct DenseGemmArgs {
  const DenseWeight* w = nullptr;
  ActOperand x;              // a batch: the operands of the matrices one after the other, each mp x kp
  int rows = 0;
  DenseSink sink = DenseSink::kPartials;
  void* out = nullptr;       // kPartials: float [splits][rows][ldo]; kRows: [rows][ldo]
  int64_t ldo = 0;
  ActOperand operand;        // kOperand
  DenseAct act = DenseAct::kNone;
  int64_t batch_cols = 0;    // column of matrix b's first feature: b * batch_cols
  int64_t n_valid = 0;       // output features stored per matrix (the rest of the last tile is dropped)
  int splits = 1;            // 1 unless kPartials
  size_t split_stride = 0;
  bool pdl = false;
};
// Rows padded the way the product's row tile wants them.
int dense_row_pad(int rows);
// How many CTAs share an output tile by splitting K (deterministic: partial sums, no atomics).
// Of two equally fast ways the one with fewer partial sums; `gain` (optional): what the split saves, in stages of
// the K loop.
int dense_splits(Precision p, int64_t n_rows, int64_t kp, int rows, int max_splits, double* gain = nullptr);
tb_status launch_dense_gemm(Precision p, const DenseGemmArgs& a, cudaStream_t st);
int dense_fault_flag();

// ---- row kernels (layered_ops.cu) --------------------------------------------------------------
// Which rows of a step belong together: row r is position pos[r] of sequence slot[r] (pos -1: dead row).
struct StepRows {
  const int32_t* tokens = nullptr;
  const int32_t* slots = nullptr;
  const int32_t* offsets = nullptr;  // as fed
  int32_t* pos = nullptr;            // offsets, -1 where token or offset is out of range (the embedding kernel writes it)
  int rows = 0;
};
// x' = source; h = norm(x') * pre_w; operand = h + causal convolution of h over time.
// Source: [norm] of the embedding (scaled table row + position row) * post_w, or x + [norm](y + bias) * post_w.
struct GlueArgs {
  StepRows r;
  // source
  DenseWeight embed;                     // embedding mode when it has an image
  float embed_scale = 1.f;
  const __nv_bfloat16* pos_table = nullptr;  // [max positions, width] or null
  int64_t vocab = 0, max_pos = 0;
  const float* x_in = nullptr;           // [rows, xs]
  PartialSums y;                         // y.y null: x' = x_in
  const float* y_bias = nullptr;         // [xs] or null
  const float* post_w = nullptr;         // [xs]; null: y is added as it is
  float* x_out = nullptr;                // [rows, xs], not x_in; null: not stored
  // sink
  const float* pre_w = nullptr;          // [xs]
  const float* conv_w = nullptr;         // [taps][xs]; null: no convolution
  int taps = 1;
  float* conv_state = nullptr;           // [slots][ring][xs], the last inputs of the convolution by position
  int ring = 0;                          // a power of two
  bool write_state = false;
  ActOperand out;                        // data null: not written
  const int32_t* row_map = nullptr;      // row -> operand row, -1: skip; null: identity
  int width = 0, xs = 0;
  float eps = 0.f;
  int row0 = 0;                          // first row handled
  bool neighbours = true;                // false: no row of the step follows another one in its sequence
  float* snapshot = nullptr;             // optional copy of x' [rows, xs]
  float* rstd = nullptr;                 // [rows] scratch: 1 / rms of x'.  When given, the glue is two kernels
                                         // (row sums, then everything per element), better for many rows;
                                         // row0 > 0 then runs the second one alone
  bool pdl = false;
};
tb_status launch_glue(Precision p, const GlueArgs& a, cudaStream_t st);

// Rows of a sequence's KV cache.  Positions below keep stay where they are, later ones live in a ring.
struct CacheGeom {
  int keep = 0;          // rows kept for the first positions
  int ring = 0;          // rows of the ring (0: row = position)
  int64_t rows = 0;      // rows per sequence
  __host__ __device__ int row_of(int pos) const { return (ring == 0 || pos < keep) ? pos : keep + (pos - keep) % ring; }
};
struct QkvPrepArgs {
  StepRows r;
  PartialSums y;
  const float* bias = nullptr;           // [ldy] or null
  const float* q_norm = nullptr;         // [q_pad] over the whole projection, or null
  const float* k_norm = nullptr;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int dpad = 0, vpad = 0;
  int q_off = 0, k_off = 0, v_off = 0;   // columns of y
  float eps = 0.f;
  float* q = nullptr;                    // [rows, heads * dpad] fp32 (or null)
  __nv_bfloat16* q16 = nullptr;          // the same in bf16 for the tensor-core kernels (or null)
  void* k_cache = nullptr;               // [slots][cache rows][kv_heads * dpad]
  void* v_cache = nullptr;               // [slots][cache rows][kv_heads * vpad]
  CacheGeom geom;
  bool pdl = false;
};
tb_status launch_qkv_prep(Precision p, const QkvPrepArgs& a, cudaStream_t st);

// Heads of a combined product [q | k | v | gates]: per-head norm of q and k without a weight, value mixing, the
// cache append, gates = sigmoid.
struct HeadsPrepArgs {
  StepRows r;
  PartialSums y;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dpad = 0, vpad = 0;
  int q_off = 0, k_off = 0, v_off = 0, g_off = 0;   // columns of y
  bool unit_norm = false;
  float eps = 0.f;
  float* v_first = nullptr;              // [rows, kv_heads * vdim] or null: v <- (1 - mix) v + mix v_first,
  bool keep_first_values = false;        // or this layer's values are the ones that later layers mix in
  float mix = 0.f;
  float* gate = nullptr;                 // [rows, heads] or null
  void* q = nullptr;                     // [rows, heads * dpad] of the activation type
  void* k_cache = nullptr;
  void* v_cache = nullptr;
  CacheGeom geom;
  bool pdl = false;
};
tb_status launch_heads_prep(Precision p, const HeadsPrepArgs& a, cudaStream_t st);

// Latent attention.  A position's cache row is [normed latent kv_rank | rotated key part rot_dim], padded to dpad; the
// query of a head lives in the same space: its unrotated part times the head's key matrix, then its rotated part.
// (q . W c = (W^T q) . c, so the keys of the heads are never written out.)
struct LatentPrepArgs {
  StepRows r;
  PartialSums y;                         // [query latent | at kv_off: key/value latent, rotated key part]
  int q_rank = 0, kv_rank = 0, rot_dim = 0, rot_dims = 0, kv_off = 0, dpad = 0;
  const float* q_norm = nullptr;         // [q_rank]
  const float* kv_norm = nullptr;        // [kv_rank]
  const float2* table = nullptr;         // [positions][rot_dims / 2] cos, sin
  float eps = 0.f;
  ActOperand out;                        // the query latent
  void* cache = nullptr;                 // [slots][cache rows][dpad]
  CacheGeom geom;
  bool pdl = false;
};
tb_status launch_latent_prep(Precision p, const LatentPrepArgs& a, cudaStream_t st);
struct LatentQueryArgs {
  StepRows r;
  PartialSums y;                         // [heads][dim | rot_dim]
  int heads = 0, dim = 0, rot_dim = 0, rot_dims = 0, dpad = 0;
  int rot_at = 0;                        // where the rotated part begins in a head's query
  const float2* table = nullptr;
  ActOperand out;                        // one operand of K = dim per head, one after the other; data null: the
                                         // unrotated part goes to the beginning of the head's query
  void* q = nullptr;                     // [rows, heads * dpad] of the activation type
  bool pdl = false;
};
tb_status launch_latent_query(Precision p, const LatentQueryArgs& a, cudaStream_t st);
// The bf16 latents of positions [lo, lo + n) of the step's first row's sequence as the operand of a product.
struct LatentRowsArgs {
  StepRows r;
  const void* cache = nullptr;           // [slots][cache rows][dpad]
  CacheGeom geom;
  int kv_rank = 0, dpad = 0;             // multiples of 8
  int lo = 0, n = 0;
  ActOperand out;
  bool pdl = false;
};
tb_status launch_latent_rows(const LatentRowsArgs& a, cudaStream_t st);
// cos and sin of position * base^(-2i / dims).
tb_status fill_rotation_table(float2* table, int64_t positions, int dims, double base);

// operand = max(z, 0)^2 (the products write it themselves when they have no partial sums)
tb_status launch_relu2(Precision p, int rows, const PartialSums& z, const ActOperand& out, bool pdl, cudaStream_t st);

// operand = a N(z) + b N(z^2) + c N(z^3) + e, N dividing a row by its root mean square (PolyNorm).
struct PolyNormArgs {
  int rows = 0;
  PartialSums z;
  int width = 0;
  float coef[4] = {0, 0, 0, 0};
  float eps = 0.f;
  ActOperand out;
  bool pdl = false;
};
tb_status launch_poly_norm(Precision p, const PolyNormArgs& a, cudaStream_t st);

// ---- attention with an online softmax (flash_attention.cu) ----------------------------------------
struct FlashArgs {
  StepRows r;
  const void* q = nullptr;               // [rows, heads * dpad] of the activation type
  const void* k_cache = nullptr;
  const void* v_cache = nullptr;
  bool values_in_keys = false;           // one key/value head whose values are the first vdim elements of its keys
  CacheGeom geom;
  int cache_slots = 0;                   // sequences that the caches hold
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dpad = 0, vpad = 0;
  float scale = 1.f;
  float softcap = 0.f;                   // 0: none
  const float* slopes = nullptr;         // [heads], taken off per position between query and key; null: none
  int window = 0;                        // position i sees j when i - j < window and i / chunk = j / chunk (chunk > 0),
  int keep_first = 0;                    // or j < keep_first
  int chunk = 0;
  bool unit_norm = false;                // queries and keys have a root mean square of one
  // Keys and values written out by position instead of the caches (portions of one sequence): position p of head g
  // is row p - key_base of key_count, its first key_cols key columns at key_rows + g key_cols, its values at value_rows + g vdim;
  // the other key columns, the same for every head, are columns from rest_col on of k_cache's rows of cache_row.
  const void* key_rows = nullptr;
  const void* value_rows = nullptr;
  int key_cols = 0, key_base = 0, key_count = 0, row_stride = 0, rest_col = 0, cache_row = 0;
  const float* gate = nullptr;           // [rows, heads] factors of the heads' outputs, or null
  int64_t max_visible = 0;               // most positions one row can see
  float* parts = nullptr;                // scratch [part_slots][vdim]
  float2* part_ml = nullptr;             // scratch [part_slots]
  int64_t part_slots = 0;
  ActOperand out;                        // K = heads * vdim
  bool out_per_head = false;             // or one operand of K = vdim per head, one after the other
  bool one_sequence = false;             // the rows are consecutive positions of one sequence
  bool pdl = false;
};
int64_t flash_part_slots(int64_t rows, int64_t heads);   // what the splits a step can use need
tb_status launch_flash_attention(Precision p, const FlashArgs& a, cudaStream_t st, int* launches);
bool flash_tc5_fits(int dpad, int vdim);                 // sizes that the tcgen05 kernel for portions takes
int flash_fault_flag();
int flash_latent_fault_flag();

// ---- windowed attention with mixed heads (window_attention.cu) -----------------------------------
struct WindowAttnArgs {
  StepRows r;
  const float* q = nullptr;              // [rows, heads * dpad]
  const __nv_bfloat16* q16 = nullptr;
  const void* k_cache = nullptr;
  const void* v_cache = nullptr;
  CacheGeom geom;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dpad = 0, vpad = 0;
  float scale = 1.f;
  int window = 0;                        // position i sees j when i - j < window or j < keep_first
  int keep_first = 0;
  const float* talk = nullptr;           // [heads][heads]
  int64_t max_visible = 0;               // most positions one row can see
  float* scores = nullptr;               // scratch [rows of a pass][heads][score_stride]
  float* part = nullptr;                 // scratch [rows of a pass][heads][splits][2]
  int64_t scratch_rows = 0;
  float* parts = nullptr;                // scratch [parts_rows][heads * vdim]: sums of CTAs that share a row's positions
  int64_t parts_rows = 0;                // rows x splits it holds
  ActOperand out;                        // K = heads * vdim
  bool one_sequence = false;             // the rows are consecutive positions of one sequence
  bool pdl = false;
};
constexpr int kScoreSplitsMax = 64;
size_t window_attn_score_stride(int64_t max_visible);
tb_status launch_window_attention(Precision p, const WindowAttnArgs& a, cudaStream_t st, int* launches);
tb_status launch_window_parts(Precision p, const WindowAttnArgs& a, int splits, int row0, int rows, cudaStream_t st);
// Tensor-core form for a portion of one sequence (window_attention_mma.cu); reads q16, not q.
bool window_mma_supported(const WindowAttnArgs& a);
tb_status launch_window_attention_mma(const WindowAttnArgs& a, cudaStream_t st, int* launches);

}  // namespace tb

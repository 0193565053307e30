// Attention with a sliding window, kept first positions and post-softmax mixing of the heads.
//
// Position i sees j when j <= i and (i - j < window or j < keep_first); the visible positions of a row are
// therefore at most two runs, and visible number v is position v < nk ? v : v - nk + lo (VisibleRange).
// The mixing  w'_h(j) = sum_g T[h, g] w_g(j)  needs every head's NORMALISED weight of a key before any of
// them meets the values, so the work is cut where the softmax is complete:
//
//   scores   raw scores of every (row, head, visible position) -> scratch, with the running (max, sum) of
//            each CTA's share of the positions
//   mix      weights = exp(score - max) / sum, mixed over the heads, times the values; a cluster of CTAs
//            shares a row's positions and adds its parts through distributed shared memory in rank order
//
// Both read the cache once.  These two serve decode steps (any number of sequences) in both precisions and
// whole portions in fp32; portions in bf16 take the tensor-core kernels in window_attention_mma.cu.
#include <cooperative_groups.h>

#include "dense.cuh"
#include "window_attention.cuh"

namespace cg = cooperative_groups;

namespace tb {

namespace {

constexpr int kThreads = 256;
constexpr int kTileP = 32;   // positions per tile: one per lane

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
  }
}
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xFFFF0000u));
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// The tile's rows (kTileP visible positions from v0) of `row_elems` elements each, into shared memory with a
// row stride of `stride` elements.  col0: first element of the cache row.
template <typename T>
__device__ __forceinline__ void stage_tile(T* s, int stride, const T* cache, int64_t cache_row, int col0, int row_elems, int v0, int nv,
                                           const VisibleRange& vr, const CacheGeom& geom) {
  constexpr int EP = 16 / sizeof(T);
  const int pieces = row_elems / EP;
  for (int i = threadIdx.x; i < kTileP * pieces; i += kThreads) {
    const int t = i / pieces, c = i - t * pieces;
    if (v0 + t < nv) cp16(s + t * stride + c * EP, cache + (size_t)geom.row_of(vr.position(v0 + t)) * cache_row + col0 + c * EP);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}

struct ScoreShape {
  int splits;       // CTAs that share a row's positions
  int kv_per;       // kv heads per CTA
  int64_t stride;   // floats per (row, head) of the score scratch
  int row0;
};

// grid (splits, kv head groups, rows)
template <typename T>
__global__ void __launch_bounds__(kThreads) window_scores_kernel(const WindowAttnArgs a, const ScoreShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads;
  const int kv0 = (int)blockIdx.y * sh.kv_per, nkv = min(sh.kv_per, a.kv_heads - kv0);
  const int h0 = kv0 * gq, nh = nkv * gq;
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  const int kcols = nkv * a.dpad, stride = kcols + 16 / (int)sizeof(T);
  float* s_q = reinterpret_cast<float*>(s_raw);
  float* s_m = s_q + sh.kv_per * gq * a.dpad;   // [nh] running max, [nh] running sum
  float* s_l = s_m + sh.kv_per * gq;
  T* s_k = reinterpret_cast<T*>(s_raw + ((sizeof(float) * (size_t)(sh.kv_per * gq) * (a.dpad + 2) + 15) & ~(size_t)15));
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first);
  const int nv = vr.count();
  const T* kc = static_cast<const T*>(a.k_cache) + (pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows * (size_t)(a.kv_heads * a.dpad));
  for (int i = tid; i < nh * a.dpad; i += kThreads) s_q[i] = a.q[(size_t)r * a.heads * a.dpad + (size_t)h0 * a.dpad + i];
  for (int i = tid; i < nh; i += kThreads) { s_m[i] = -INFINITY; s_l[i] = 0.f; }
  const int tiles = (nv + kTileP - 1) / kTileP;
  const int t0 = (int)((int64_t)tiles * blockIdx.x / sh.splits), t1 = (int)((int64_t)tiles * (blockIdx.x + 1) / sh.splits);
  for (int t = t0; t < t1; ++t) {
    __syncthreads();
    stage_tile(s_k, stride, kc, a.kv_heads * a.dpad, kv0 * a.dpad, kcols, t * kTileP, nv, vr, a.geom);
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const int v = t * kTileP + lane;
    for (int h = warp; h < nh; h += kThreads / 32) {
      const T* kr = s_k + lane * stride + (h / gq) * a.dpad;
      const float* q = s_q + h * a.dpad;
      float acc0 = 0.f, acc1 = 0.f;
      if (v < nv) {
        for (int c = 0; c < a.dpad; c += 8) {
          float k8[8];
          load8<T>(kr + c, k8);
          const float4 qa = *reinterpret_cast<const float4*>(q + c), qb = *reinterpret_cast<const float4*>(q + c + 4);
          acc0 = fmaf(qa.x, k8[0], acc0); acc1 = fmaf(qa.y, k8[1], acc1);
          acc0 = fmaf(qa.z, k8[2], acc0); acc1 = fmaf(qa.w, k8[3], acc1);
          acc0 = fmaf(qb.x, k8[4], acc0); acc1 = fmaf(qb.y, k8[5], acc1);
          acc0 = fmaf(qb.z, k8[6], acc0); acc1 = fmaf(qb.w, k8[7], acc1);
        }
      }
      const float s = v < nv ? (acc0 + acc1) * a.scale : -INFINITY;
      if (v < nv) a.scores[((size_t)lr * a.heads + h0 + h) * sh.stride + v] = s;
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      float l = v < nv ? expf(s - mx) : 0.f;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      if (lane == 0) {
        const float m0 = s_m[h], m1 = fmaxf(m0, mx);
        s_l[h] = (m0 == -INFINITY ? 0.f : s_l[h] * expf(m0 - m1)) + l * expf(mx - m1);
        s_m[h] = m1;
      }
    }
  }
  __syncthreads();
  for (int h = tid; h < nh; h += kThreads) {
    float* p = a.part + (((size_t)lr * a.heads + h0 + h) * sh.splits + blockIdx.x) * 2;
    p[0] = s_m[h];
    p[1] = s_l[h];
  }
}

// grid (cluster size, head blocks, rows); hb heads per CTA
template <typename T, bool BF16>
__global__ void __launch_bounds__(kThreads) window_mix_kernel(const WindowAttnArgs a, const ScoreShape sh, const int hb, const int kvs) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads;
  const int h0 = (int)blockIdx.y * hb, nh = min(hb, a.heads - h0);
  const int kv0 = h0 / gq, nkv = (h0 + nh - 1) / gq - kv0 + 1;
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  const int vcols = nkv * a.vpad, stride = kvs * a.vpad + 16 / (int)sizeof(T);
  float* s_m = reinterpret_cast<float*>(s_raw);           // [heads]
  float* s_il = s_m + a.heads;                            // [heads]
  float* s_t = s_il + a.heads;                            // [hb][heads]
  float* s_p = s_t + hb * a.heads;                        // [heads][kTileP]
  float* s_w = s_p + a.heads * kTileP;                    // [hb][kTileP]
  float* s_acc = s_w + hb * kTileP;                       // [hb][vpad]
  const size_t fl = (size_t)a.heads * 2 + (size_t)hb * a.heads + (size_t)a.heads * kTileP + (size_t)hb * kTileP + (size_t)hb * a.vpad;
  T* s_v = reinterpret_cast<T*>(s_raw + ((fl * sizeof(float) + 15) & ~(size_t)15));
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int csize = (int)gridDim.x, crank = (int)blockIdx.x;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first);
  const int nv = vr.count();
  const T* vc = static_cast<const T*>(a.v_cache) + (pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows * (size_t)(a.kv_heads * a.vpad));
  for (int g = warp; g < a.heads; g += kThreads / 32) {   // softmax statistics from the parts, in order
    const float* p = a.part + ((size_t)lr * a.heads + g) * sh.splits * 2;
    float m = -INFINITY;
    for (int s = lane; s < sh.splits; s += 32) m = fmaxf(m, p[2 * s]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float l = 0.f;
    for (int s = lane; s < sh.splits; s += 32) l += p[2 * s] == -INFINITY ? 0.f : p[2 * s + 1] * expf(p[2 * s] - m);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (lane == 0) { s_m[g] = m; s_il[g] = l > 0.f ? 1.0f / l : 0.f; }
  }
  for (int i = tid; i < nh * a.heads; i += kThreads) s_t[i] = a.talk[(size_t)h0 * a.heads + i];
  for (int i = tid; i < nh * a.vpad; i += kThreads) s_acc[i] = 0.f;
  const int tiles = (nv + kTileP - 1) / kTileP;
  const int t0 = (int)((int64_t)tiles * crank / csize), t1 = (int)((int64_t)tiles * (crank + 1) / csize);
  for (int t = t0; t < t1; ++t) {
    __syncthreads();
    stage_tile(s_v, stride, vc, a.kv_heads * a.vpad, kv0 * a.vpad, vcols, t * kTileP, nv, vr, a.geom);
    const int v = t * kTileP + lane;
    for (int g = warp; g < a.heads; g += kThreads / 32)
      s_p[g * kTileP + lane] = v < nv ? expf(a.scores[((size_t)lr * a.heads + g) * sh.stride + v] - s_m[g]) * s_il[g] : 0.f;
    __syncthreads();
    for (int h = warp; h < nh; h += kThreads / 32) {
      const float* tr = s_t + h * a.heads;
      float w0 = 0.f, w1 = 0.f;
      int g = 0;
      for (; g + 1 < a.heads; g += 2) {
        w0 = fmaf(tr[g], s_p[g * kTileP + lane], w0);
        w1 = fmaf(tr[g + 1], s_p[(g + 1) * kTileP + lane], w1);
      }
      if (g < a.heads) w0 = fmaf(tr[g], s_p[g * kTileP + lane], w0);
      s_w[h * kTileP + lane] = w0 + w1;
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const int nt = min(kTileP, nv - t * kTileP);
    const int c2 = a.vpad >> 1;
    for (int i = tid; i < nh * c2; i += kThreads) {   // (head, pair of columns)
      const int h = i / c2, c = (i - h * c2) * 2;
      const T* vp = s_v + ((h0 + h) / gq - kv0) * a.vpad + c;
      const float* w = s_w + h * kTileP;
      float2 acc = make_float2(0.f, 0.f);
#pragma unroll 8
      for (int j = 0; j < nt; ++j) {
        const float2 x = load2(vp + j * stride);
        acc.x = fmaf(w[j], x.x, acc.x);
        acc.y = fmaf(w[j], x.y, acc.y);
      }
      s_acc[h * a.vpad + c] += acc.x;
      s_acc[h * a.vpad + c + 1] += acc.y;
    }
  }
  // sum over the cluster in rank order; every CTA finishes a slice of the columns
  cg::cluster_group cl = cg::this_cluster();
  if (csize > 1) cl.sync();
  else __syncthreads();
  const int total = nh * a.vdim, per = (total + csize - 1) / csize;
  for (int i = crank * per + tid; i < min(total, (crank + 1) * per); i += kThreads) {
    const int h = i / a.vdim, c = i - h * a.vdim;
    float v = 0.f;
    if (csize > 1) {
      for (int q = 0; q < csize; ++q) v += *cl.map_shared_rank(&s_acc[h * a.vpad + c], q);
    } else {
      v = s_acc[h * a.vpad + c];
    }
    act_store1<BF16>(a.out, r, (h0 + h) * a.vdim + c, pos < 0 ? 0.f : v);
  }
  if (h0 + nh == a.heads && crank == 0)
    for (int k = a.heads * a.vdim + tid; k < a.out.kp; k += kThreads) act_store1<BF16>(a.out, r, k, 0.f);
  if (csize > 1) cl.sync();   // nobody leaves while its sums may still be read
}

template <typename T, bool BF16>
tb_status launch_generic(const WindowAttnArgs& a, cudaStream_t st, int* launches) {
  const int gq = a.heads / a.kv_heads;
  const size_t lim = 96 * 1024;
  ScoreShape sh;
  sh.stride = (int64_t)window_attn_score_stride(a.max_visible);
  // scores: kv heads per CTA so that a tile and the queries fit
  auto sbytes = [&](int kv) {
    return ((sizeof(float) * (size_t)(kv * gq) * (a.dpad + 2) + 15) & ~(size_t)15) + (size_t)kTileP * (kv * a.dpad + 16 / sizeof(T)) * sizeof(T);
  };
  int kv = a.kv_heads;
  while (kv > 1 && sbytes(kv) > lim) kv = (kv + 1) / 2;
  sh.kv_per = kv;
  const int kgroups = (a.kv_heads + kv - 1) / kv;
  // mix: heads per CTA
  int kvs = 1;
  auto mbytes = [&](int hb) {
    const size_t fl = (size_t)a.heads * 2 + (size_t)hb * a.heads + (size_t)a.heads * kTileP + (size_t)hb * kTileP + (size_t)hb * a.vpad;
    kvs = (hb + gq - 2) / gq + 1;   // most kv heads a block of hb heads touches
    if (hb % gq == 0) kvs = hb / gq;
    else if (gq % hb == 0) kvs = 1;
    if (kvs > a.kv_heads) kvs = a.kv_heads;
    return ((fl * sizeof(float) + 15) & ~(size_t)15) + (size_t)kTileP * (kvs * a.vpad + 16 / sizeof(T)) * sizeof(T);
  };
  const int64_t tiles = (a.max_visible + kTileP - 1) / kTileP;
  int64_t pass = a.r.rows < a.scratch_rows ? a.r.rows : a.scratch_rows;
  if (pass > 32768) pass = 32768;
  const int rows_like = (int)pass;
  // CTAs that share a row: scores split freely, mix in a cluster
  int splits = (2 * sm_count() + rows_like * kgroups - 1) / (rows_like * kgroups);
  if (splits > tiles) splits = (int)tiles;
  if (splits > kScoreSplitsMax) splits = kScoreSplitsMax;
  if (splits < 1) splits = 1;
  sh.splits = splits;
  int cluster = 1;
  while (cluster < 8 && cluster * 2 <= tiles && rows_like * cluster * 2 <= 2 * sm_count()) cluster *= 2;
  int hb = a.heads;
  while (hb > 1 && (mbytes(hb) > lim || (int64_t)rows_like * cluster * ((a.heads + hb - 1) / hb) < sm_count() * 3 / 4)) hb = (hb + 1) / 2;
  const size_t msm = mbytes(hb);
  if (sbytes(kv) > 200 * 1024 || msm > 200 * 1024)
    return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: attention with %d heads of size %d/%d", a.heads, a.dim, a.vdim);
  const int hblocks = (a.heads + hb - 1) / hb;
  for (int64_t r0 = 0; r0 < a.r.rows; r0 += pass) {
    const int n = (int)(a.r.rows - r0 < pass ? a.r.rows - r0 : pass);
    sh.row0 = (int)r0;
    TB_TRY(launch_kernel(window_scores_kernel<T>, dim3((unsigned)splits, (unsigned)kgroups, (unsigned)n), dim3(kThreads), sbytes(kv), st, a.pdl, 1, a, sh));
    TB_TRY(launch_kernel(window_mix_kernel<T, BF16>, dim3((unsigned)cluster, (unsigned)hblocks, (unsigned)n), dim3(kThreads), msm, st, a.pdl, cluster,
                         a, sh, hb, kvs));
    *launches += 2;
  }
  return TB_OK;
}

}  // namespace

size_t window_attn_score_stride(int64_t max_visible) {
  // the tensor-core form numbers keys per block of 64 queries: up to 63 more than one row sees
  return (size_t)pad_to(max_visible + 64, 32);
}

tb_status launch_window_attention(Precision p, const WindowAttnArgs& a, cudaStream_t st, int* launches) {
  if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dpad % 16 || a.vpad % 16 || a.scratch_rows < 1)
    return fail(TB_ERR_SHAPE, "window attention: bad shape");
  if (p == Precision::kBf16 && window_mma_supported(a)) return launch_window_attention_mma(a, st, launches);
  if (p == Precision::kBf16) return launch_generic<__nv_bfloat16, true>(a, st, launches);
  return launch_generic<float, false>(a, st, launches);
}

}  // namespace tb

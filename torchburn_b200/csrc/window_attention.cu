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

constexpr int kTileP = 32;        // positions per tile: one per lane
constexpr int kMixThreads = 512;  // one thread per position in the weight phase of the mix kernel
constexpr int kMixWarps = kMixThreads / 32;
constexpr int kHeadChunk = 4;     // query heads that share a key's load

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

struct ScoreShape {
  int splits;       // CTAs that share a row's positions
  int64_t stride;   // floats per (row, head) of the score scratch
  int row0;
};

// grid (splits, kv heads, rows).  A warp takes 32 positions at a time: their keys by cp.async into the warp's own
// tile, then one position per lane against every query head of the kv head.
template <typename T>
__global__ void __launch_bounds__(256) window_scores_kernel(const WindowAttnArgs a, const ScoreShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  constexpr int EP = 16 / (int)sizeof(T);
  const int gq = a.heads / a.kv_heads;
  const int kv = (int)blockIdx.y, h0 = kv * gq;
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  const int stride = a.dpad + EP, pieces = a.dpad / EP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = (int)blockDim.x >> 5;
  float* s_q = reinterpret_cast<float*>(s_raw);        // [gq][dpad]
  float2* s_ml = reinterpret_cast<float2*>(s_q + gq * a.dpad);   // [warps][gq] running (max, sum)
  T* s_k = reinterpret_cast<T*>(s_raw + (((size_t)gq * a.dpad * 4 + (size_t)nw * gq * 8 + 15) & ~(size_t)15)) + (size_t)warp * kTileP * stride;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first);
  const int nv = vr.count();
  const int64_t crow_elems = (int64_t)a.kv_heads * a.dpad;
  const T* kc = static_cast<const T*>(a.k_cache) + (pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows * crow_elems) + kv * a.dpad;
  const int tiles = (nv + kTileP - 1) / kTileP;
  const int t0 = (int)((int64_t)tiles * blockIdx.x / sh.splits), t1 = (int)((int64_t)tiles * (blockIdx.x + 1) / sh.splits);
  auto stage = [&](int t) {
    const int v = t * kTileP + lane;
    const int crow = a.geom.row_of(vr.position(v < nv ? v : nv - 1));
    int tr = lane / pieces, c = lane - tr * pieces;
    const int rstep = 32 / pieces, cstep = 32 - rstep * pieces;
    for (int i = 0; i < pieces; ++i) {   // 32 * pieces copies, 32 at a time
      const int src = __shfl_sync(0xffffffffu, crow, tr);
      cp16(s_k + tr * stride + c * EP, kc + (size_t)src * crow_elems + c * EP);
      tr += rstep;
      c += cstep;
      if (c >= pieces) { c -= pieces; ++tr; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 + warp < t1) stage(t0 + warp);
  for (int i = tid; i < gq * a.dpad; i += (int)blockDim.x) s_q[i] = a.q[(size_t)r * a.heads * a.dpad + (size_t)h0 * a.dpad + i];
  for (int i = tid; i < nw * gq; i += (int)blockDim.x) s_ml[i] = make_float2(-INFINITY, 0.f);
  __syncthreads();
  for (int t = t0 + warp; t < t1; t += nw) {
    if (t != t0 + warp) stage(t);
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncwarp();
    const int v = t * kTileP + lane;
    const T* kr = s_k + lane * stride;
    for (int hb = 0; hb < gq; hb += kHeadChunk) {
      float acc[kHeadChunk];
#pragma unroll
      for (int j = 0; j < kHeadChunk; ++j) acc[j] = 0.f;
      const float* q = s_q + hb * a.dpad;
#pragma unroll 2
      for (int c = 0; c < a.dpad; c += 8) {
        float k8[8];
        load8<T>(kr + c, k8);
#pragma unroll
        for (int j = 0; j < kHeadChunk; ++j) {
          if (hb + j < gq) {
            const float4 qa = *reinterpret_cast<const float4*>(q + j * a.dpad + c), qb = *reinterpret_cast<const float4*>(q + j * a.dpad + c + 4);
            acc[j] = fmaf(qa.x, k8[0], fmaf(qa.y, k8[1], fmaf(qa.z, k8[2], fmaf(qa.w, k8[3], acc[j]))));
            acc[j] = fmaf(qb.x, k8[4], fmaf(qb.y, k8[5], fmaf(qb.z, k8[6], fmaf(qb.w, k8[7], acc[j]))));
          }
        }
      }
#pragma unroll
      for (int j = 0; j < kHeadChunk; ++j) {
        if (hb + j >= gq) break;
        const int h = hb + j;
        const float s = v < nv ? acc[j] * a.scale : -INFINITY;
        if (v < nv) a.scores[((size_t)lr * a.heads + h0 + h) * sh.stride + v] = s;
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float l = v < nv ? expf(s - mx) : 0.f;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        if (lane == 0) {
          const float2 old = s_ml[warp * gq + h];
          const float m1 = fmaxf(old.x, mx);
          s_ml[warp * gq + h] = make_float2(m1, (old.x == -INFINITY ? 0.f : old.y * expf(old.x - m1)) + l * expf(mx - m1));
        }
      }
    }
    __syncwarp();
  }
  __syncthreads();
  for (int h = tid; h < gq; h += (int)blockDim.x) {
    float m = -INFINITY, l = 0.f;
    for (int w = 0; w < nw; ++w) m = fmaxf(m, s_ml[w * gq + h].x);
    for (int w = 0; w < nw; ++w) {
      const float2 p = s_ml[w * gq + h];
      if (p.x != -INFINITY) l += p.y * expf(p.x - m);
    }
    float* p = a.part + (((size_t)lr * a.heads + h0 + h) * sh.splits + blockIdx.x) * 2;
    p[0] = m;
    p[1] = l;
  }
}

// grid (cluster size, head groups, rows): HG query heads of one kv head per CTA.  512 positions at a time: a
// thread takes one position through all heads (weights and mixing, in registers), then a warp takes 32 of the
// positions, its lanes the value columns.
template <typename T, bool BF16, int HG>
__global__ void __launch_bounds__(kMixThreads, 1) window_mix_kernel(const WindowAttnArgs a, const ScoreShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads, per_kv = (gq + HG - 1) / HG;
  const int kv = (int)blockIdx.y / per_kv, sub = (int)blockIdx.y - kv * per_kv;
  const int h0 = kv * gq + sub * HG, nh = min(HG, gq - sub * HG);
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  float* s_m = reinterpret_cast<float*>(s_raw);                                // [heads]
  float* s_il = s_m + a.heads;                                                 // [heads]
  float* s_t = reinterpret_cast<float*>(s_raw + (((size_t)a.heads * 8 + 15) & ~(size_t)15));   // [heads][HG]
  float* s_w = s_t + (((size_t)a.heads * HG + 3) & ~(size_t)3);                // [512][HG]
  float* s_red = s_w + kMixThreads * HG;                                       // [warps][HG][vpad]
  float* s_acc = s_red + (size_t)kMixWarps * HG * a.vpad;                      // [HG][vpad]
  int* s_row = reinterpret_cast<int*>(s_acc + HG * a.vpad);                    // [512] cache rows
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int csize = (int)gridDim.x, crank = (int)blockIdx.x;
  grid_dep_launch();
  for (int i = tid; i < a.heads * HG; i += kMixThreads) {
    const int g = i / HG, h = i - g * HG;
    s_t[i] = h < nh ? a.talk[(size_t)(h0 + h) * a.heads + g] : 0.f;
  }
  for (int i = lane; i < HG * a.vpad; i += 32) s_red[(size_t)warp * HG * a.vpad + i] = 0.f;
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first);
  const int nv = vr.count();
  const int64_t crow_elems = (int64_t)a.kv_heads * a.vpad;
  const T* vc = static_cast<const T*>(a.v_cache) + (pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows * crow_elems) + kv * a.vpad;
  for (int g = warp; g < a.heads; g += kMixWarps) {   // softmax statistics from the parts, in a fixed order
    const float2* p = reinterpret_cast<const float2*>(a.part) + ((size_t)lr * a.heads + g) * sh.splits;
    const float2 p0 = lane < sh.splits ? p[lane] : make_float2(-INFINITY, 0.f);
    const float2 p1 = lane + 32 < sh.splits ? p[lane + 32] : make_float2(-INFINITY, 0.f);
    float m = fmaxf(p0.x, p1.x);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float l = (p0.x == -INFINITY ? 0.f : p0.y * expf(p0.x - m)) + (p1.x == -INFINITY ? 0.f : p1.y * expf(p1.x - m));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (lane == 0) { s_m[g] = m; s_il[g] = l > 0.f ? 1.0f / l : 0.f; }
  }
  __syncthreads();
  // this CTA's positions, in blocks of 512
  const int v_begin = (int)((int64_t)nv * crank / csize), v_end = (int)((int64_t)nv * (crank + 1) / csize);
  for (int v0 = v_begin; v0 < v_end; v0 += kMixThreads) {
    const int v = v0 + tid;
    const bool live = v < v_end;
    const float* sp = a.scores + (size_t)lr * a.heads * sh.stride + (live ? v : v0);
    float w[HG];
#pragma unroll
    for (int h = 0; h < HG; ++h) w[h] = 0.f;
    constexpr int GB = 8;
    for (int g0 = 0; g0 < a.heads; g0 += GB) {
      float s8[GB];
#pragma unroll
      for (int j = 0; j < GB; ++j) s8[j] = g0 + j < a.heads ? sp[(size_t)(g0 + j) * sh.stride] : 0.f;
#pragma unroll
      for (int j = 0; j < GB; ++j) {
        const int g = g0 + j;
        if (g < a.heads) {
          const float p = expf(s8[j] - s_m[g]) * s_il[g];
#pragma unroll
          for (int h = 0; h < HG; ++h) w[h] = fmaf(s_t[g * HG + h], p, w[h]);
        }
      }
    }
    if (live) {
#pragma unroll
      for (int h = 0; h < HG; ++h) s_w[tid * HG + h] = w[h];
      s_row[tid] = a.geom.row_of(vr.position(v));
    }
    __syncthreads();
    const int j0 = warp * 32, nj = min(32, v_end - v0 - j0);
    if (nj > 0)
      for (int c = lane * 2; c < a.vpad; c += 64) {
        float2 acc[HG];
#pragma unroll
        for (int h = 0; h < HG; ++h) acc[h] = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int j = 0; j < nj; ++j) {
          const float2 x = load2(vc + (size_t)s_row[j0 + j] * crow_elems + c);
#pragma unroll
          for (int h = 0; h < HG; ++h) {
            const float wj = s_w[(j0 + j) * HG + h];
            acc[h].x = fmaf(wj, x.x, acc[h].x);
            acc[h].y = fmaf(wj, x.y, acc[h].y);
          }
        }
        float* d = s_red + (size_t)warp * HG * a.vpad + c;
#pragma unroll
        for (int h = 0; h < HG; ++h) {
          d[h * a.vpad] += acc[h].x;
          d[h * a.vpad + 1] += acc[h].y;
        }
      }
    __syncthreads();
  }
  __syncthreads();
  for (int i = tid; i < HG * a.vpad; i += kMixThreads) {
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < kMixWarps; ++q) v += s_red[(size_t)q * HG * a.vpad + i];
    s_acc[i] = v;
  }
  // sum over the cluster in rank order; every CTA finishes a slice of the columns
  cg::cluster_group cl = cg::this_cluster();
  if (csize > 1) cl.sync();
  else __syncthreads();
  const int total = nh * a.vdim, per = (total + csize - 1) / csize;
  for (int i = crank * per + tid; i < min(total, (crank + 1) * per); i += kMixThreads) {
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
    for (int k = a.heads * a.vdim + tid; k < a.out.kp; k += kMixThreads) act_store1<BF16>(a.out, r, k, 0.f);
  if (csize > 1) cl.sync();   // nobody leaves while its sums may still be read
}

template <typename T, bool BF16>
tb_status launch_generic(const WindowAttnArgs& a, cudaStream_t st, int* launches) {
  const int gq = a.heads / a.kv_heads;
  ScoreShape sh;
  sh.stride = (int64_t)window_attn_score_stride(a.max_visible);
  const int64_t tiles = (a.max_visible + kTileP - 1) / kTileP;
  int64_t pass = a.r.rows < a.scratch_rows ? a.r.rows : a.scratch_rows;
  if (pass > 32768) pass = 32768;
  const int64_t rows = pass;
  // scores: as many warps as their tiles fit
  auto sbytes = [&](int w) {
    return (((size_t)gq * a.dpad * 4 + (size_t)w * gq * 8 + 15) & ~(size_t)15) + (size_t)w * kTileP * (a.dpad + 16 / sizeof(T)) * sizeof(T);
  };
  int warps = 8;
  while (warps > 1 && (sbytes(warps) > 112 * 1024 || warps / 2 >= tiles)) warps /= 2;
  int64_t splits = (2 * sm_count() + rows * a.kv_heads - 1) / (rows * a.kv_heads);
  if (splits > (tiles + warps - 1) / warps) splits = (tiles + warps - 1) / warps;
  if (splits > kScoreSplitsMax) splits = kScoreSplitsMax;
  sh.splits = (int)splits;
  // mix: query heads of one kv head per CTA, a cluster over the positions
  const int hg = gq >= 4 ? 4 : (gq >= 2 ? 2 : 1);
  const int groups = a.kv_heads * ((gq + hg - 1) / hg);
  int cluster = 1;
  while (cluster < 8 && (int64_t)cluster * 64 < a.max_visible && rows * groups * cluster < sm_count()) cluster *= 2;
  const size_t msm = (((size_t)a.heads * 8 + 15) & ~(size_t)15) +
                     4 * ((((size_t)a.heads * hg + 3) & ~(size_t)3) + (size_t)kMixThreads * hg + (size_t)(kMixWarps + 1) * hg * a.vpad + kMixThreads);
  if (sbytes(warps) > 200 * 1024 || msm > 200 * 1024)
    return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: attention with %d heads of size %d/%d", a.heads, a.dim, a.vdim);
  auto* mix = hg == 4 ? window_mix_kernel<T, BF16, 4> : (hg == 2 ? window_mix_kernel<T, BF16, 2> : window_mix_kernel<T, BF16, 1>);
  for (int64_t r0 = 0; r0 < a.r.rows; r0 += pass) {
    const int n = (int)(a.r.rows - r0 < pass ? a.r.rows - r0 : pass);
    sh.row0 = (int)r0;
    TB_TRY(launch_kernel(window_scores_kernel<T>, dim3((unsigned)sh.splits, (unsigned)a.kv_heads, (unsigned)n), dim3((unsigned)warps * 32),
                         sbytes(warps), st, a.pdl, 1, a, sh));
    TB_TRY(launch_kernel(mix, dim3((unsigned)cluster, (unsigned)groups, (unsigned)n), dim3(kMixThreads), msm, st, a.pdl, cluster, a, sh));
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

// Attention with a sliding window, kept first positions and post-softmax mixing of the heads.
//
// Position i sees j when j <= i and (i - j < window or j < keep_first); the visible positions of a row are
// therefore at most two runs, and visible number v is position v < nk ? v : v - nk + lo (VisibleRange).
// The mixing  w'_h(j) = sum_g T[h, g] w_g(j)  needs every head's NORMALISED weight of a key before any of
// them meets the values, so the work is cut where the softmax is complete:
//
//   scores   raw scores of every (row, head, visible position) -> scratch, with the running (max, sum) of
//            each CTA's share of the positions
//   mix      weights = exp(score - max) / sum, mixed over the heads, times the values.  The weights are
//            normalised, so CTAs that share a row's positions leave plain sums, added in order by a last kernel
//
// Each half of the cache is read once.  These two serve decode steps (any number of sequences) in both precisions and
// whole portions in fp32; portions in bf16 take the tensor-core kernels in window_attention_mma.cu.
#include "dense.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

constexpr int kTileP = 32;        // positions per tile: one per lane
constexpr int kMixThreads = 256;
constexpr float kLog2E = 1.44269504f;
constexpr int kHeadChunk = 4;     // query heads that share a key's load

__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xFFFF0000u));
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct ScoreShape {
  int splits;       // CTAs that share a row's positions
  int64_t stride;   // floats per (row, head) of the score scratch
  int row0, rows;   // rows of this pass
};

// Bytes of the queries of one kv head in shared memory.  fp32: [heads][dpad].  bf16: per four heads eight rows
// [dpad + 8]: the heads rounded to bf16, then what the rounding left (together 16 mantissa bits).
template <typename T>
__host__ __device__ constexpr size_t query_bytes(int gq, int dpad) {
  return sizeof(T) == 4 ? (size_t)gq * dpad * 4 : (size_t)((gq + 3) / 4) * 8 * (dpad + 8) * 2;
}

// grid (splits, kv heads, rows).  A warp takes 32 positions at a time, their keys by cp.async into the warp's own
// tile.  fp32: one position per lane against every query head of the kv head.  bf16: the keys are the 16-row side
// of mma.sync, the two pieces of four query heads its eight columns.
template <typename T>
__global__ void __launch_bounds__(256) window_scores_kernel(const WindowAttnArgs a, const ScoreShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  constexpr int EP = 16 / (int)sizeof(T);
  constexpr bool MMA = sizeof(T) == 2;
  const int gq = a.heads / a.kv_heads;
  const int kv = (int)blockIdx.y, h0 = kv * gq;
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  const int stride = a.dpad + EP, pieces = a.dpad / EP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = (int)blockDim.x >> 5;
  const size_t qb = query_bytes<T>(gq, a.dpad);
  float2* s_ml = reinterpret_cast<float2*>(s_raw + qb);   // [warps][gq] running (max, sum)
  T* s_k = reinterpret_cast<T*>(s_raw + ((qb + (size_t)nw * gq * 8 + 15) & ~(size_t)15)) + (size_t)warp * kTileP * stride;
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
      cp16(s_k + tr * stride + c * EP, kc + (size_t)(uint32_t)src * (uint32_t)crow_elems + c * EP);
      tr += rstep;
      c += cstep;
      if (c >= pieces) { c -= pieces; ++tr; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 + warp < t1) stage(t0 + warp);
  const float* qrow = a.q + (size_t)r * a.heads * a.dpad + (size_t)h0 * a.dpad;
  if constexpr (MMA) {
    __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(s_raw);
    for (int i = tid; i < (gq + 3) / 4 * 4 * a.dpad; i += (int)blockDim.x) {
      const int h = i / a.dpad, c = i - h * a.dpad;
      const float q = h < gq ? qrow[i] : 0.f;
      const __nv_bfloat16 hi = __float2bfloat16_rn(q);
      __nv_bfloat16* d = s_q + (size_t)((h >> 2) * 8 + (h & 3)) * (a.dpad + 8) + c;
      d[0] = hi;
      d[4 * (a.dpad + 8)] = __float2bfloat16_rn(q - __bfloat162float(hi));
    }
  } else {
    float* s_q = reinterpret_cast<float*>(s_raw);
    for (int i = tid; i < gq * a.dpad; i += (int)blockDim.x) s_q[i] = qrow[i];
  }
  for (int i = tid; i < nw * gq; i += (int)blockDim.x) s_ml[i] = make_float2(-INFINITY, 0.f);
  __syncthreads();
  // running (max, sum) of head h with the maximum and sum of a tile
  auto fold = [&](int h, float mx, float l) {
    const float2 old = s_ml[warp * gq + h];
    const float m1 = fmaxf(old.x, mx);
    s_ml[warp * gq + h] = make_float2(m1, (old.x == -INFINITY ? 0.f : old.y * expf(old.x - m1)) + l * expf(mx - m1));
  };
  float* srow = a.scores + ((size_t)lr * a.heads + h0) * sh.stride;
  for (int t = t0 + warp; t < t1; t += nw) {
    if (t != t0 + warp) stage(t);
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncwarp();
    for (int hb = 0; hb < gq; hb += kHeadChunk) {
      if constexpr (MMA) {
        const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(s_raw) + (size_t)((hb >> 2) * 8 + (lane >> 2)) * (a.dpad + 8) + (lane & 3) * 2;
        float d[2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int i = 0; i < 4; ++i) d[m][i] = 0.f;
#pragma unroll 4
        for (int c = 0; c < a.dpad; c += 16) {
          const uint32_t b0 = *reinterpret_cast<const uint32_t*>(q + c), b1 = *reinterpret_cast<const uint32_t*>(q + c + 8);
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            uint32_t ka[4];
            ldm4(ka, s_k + (m * 16 + (lane & 15)) * stride + c + (lane >> 4) * 8);
            mma16816(d[m], ka, b0, b1);
          }
        }
        // d[m][2 x + y]: position 16 m + lane / 4 + 8 x, column 2 (lane & 3) + y = piece (lane & 3) / 2 of head 2 (lane & 1) + y
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int i = 0; i < 4; ++i) d[m][i] += __shfl_xor_sync(0xffffffffu, d[m][i], 2);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int h = hb + (lane & 1) * 2 + y;
          float s[4], mx = -INFINITY;
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int v = t * kTileP + (x >> 1) * 16 + (lane >> 2) + (x & 1) * 8;
            s[x] = v < nv ? d[x >> 1][(x & 1) * 2 + y] * a.scale : -INFINITY;
            if (v < nv && (lane & 2) == 0 && h < gq) srow[(size_t)h * sh.stride + v] = s[x];
            mx = fmaxf(mx, s[x]);
          }
#pragma unroll
          for (int o = 16; o > 2; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
          float l = 0.f;
#pragma unroll
          for (int x = 0; x < 4; ++x) l += expf(s[x] - mx);
#pragma unroll
          for (int o = 16; o > 2; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
          if (lane < 2 && h < gq) fold(h, mx, l);
        }
      } else {
        const int v = t * kTileP + lane;
        const T* kr = s_k + lane * stride;
        float acc[kHeadChunk];
#pragma unroll
        for (int j = 0; j < kHeadChunk; ++j) acc[j] = 0.f;
        const float* q = reinterpret_cast<const float*>(s_raw) + hb * a.dpad;
#pragma unroll 2
        for (int c = 0; c < a.dpad; c += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kr + c);
#pragma unroll
          for (int j = 0; j < kHeadChunk; ++j) {
            if (hb + j < gq) {
              const float4 q4 = *reinterpret_cast<const float4*>(q + j * a.dpad + c);
              acc[j] = fmaf(q4.x, k4.x, fmaf(q4.y, k4.y, fmaf(q4.z, k4.z, fmaf(q4.w, k4.w, acc[j]))));
            }
          }
        }
#pragma unroll
        for (int j = 0; j < kHeadChunk; ++j) {
          if (hb + j >= gq) break;
          const float s = v < nv ? acc[j] * a.scale : -INFINITY;
          if (v < nv) srow[(size_t)(hb + j) * sh.stride + v] = s;
          float mx = s;
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
          float l = v < nv ? expf(s - mx) : 0.f;
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
          if (lane == 0) fold(hb + j, mx, l);
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

template <int N>
__device__ __forceinline__ void load_row(const float* p, float (&v)[N]) {   // p aligned to the row
  if constexpr (N == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  } else if constexpr (N == 2) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    v[0] = x.x; v[1] = x.y;
  } else {
    v[0] = *p;
  }
}

// A warp's 32 positions times the values: lanes own CPL neighbouring columns; sums are added to `red` (the warp's own).
template <typename T, int HG, int CPL>
__device__ __forceinline__ void warp_values(const T* vals, const int* rows, int64_t row_elems, const float* w, int nj, int vpad, float* red) {
  const int lane = threadIdx.x & 31;
  for (int c = lane * CPL; c < vpad; c += 32 * CPL) {
    float acc[HG][CPL];
#pragma unroll
    for (int h = 0; h < HG; ++h)
#pragma unroll
      for (int i = 0; i < CPL; ++i) acc[h][i] = 0.f;
#pragma unroll 8
    for (int j = 0; j < nj; ++j) {
      const T* p = vals + (size_t)(rows ? rows[j] : j) * row_elems + c;
      float x[CPL];
#pragma unroll
      for (int i = 0; i < CPL; i += 2) {
        const float2 f = load2(p + i);
        x[i] = f.x;
        x[i + 1] = f.y;
      }
      float wj[HG];
      load_row<HG>(w + j * HG, wj);
#pragma unroll
      for (int h = 0; h < HG; ++h)
#pragma unroll
        for (int i = 0; i < CPL; ++i) acc[h][i] = fmaf(wj[h], x[i], acc[h][i]);
    }
#pragma unroll
    for (int h = 0; h < HG; ++h)
#pragma unroll
      for (int i = 0; i < CPL; ++i) red[h * vpad + c + i] += acc[h][i];
  }
}

// grid (position splits, head groups, rows): HG query heads of one kv head per CTA.  A warp takes 32 positions at a
// time and needs no other: their values by cp.async into the warp's tile (VSM) while a lane takes one position
// through all heads (weights and mixing, in registers), then the lanes are the value columns.
// VSM: 0 values from global memory, 1 staged, fp32 products, 2 staged, mma.sync (bf16, at most 128 columns).
template <typename T, bool BF16, int HG, int VSM>
__global__ void __launch_bounds__(kMixThreads, 2) window_mix_kernel(const WindowAttnArgs a, const ScoreShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads, per_kv = (gq + HG - 1) / HG;
  const int kv = (int)blockIdx.y / per_kv, sub = (int)blockIdx.y - kv * per_kv;
  const int h0 = kv * gq + sub * HG, nh = min(HG, gq - sub * HG);
  const int lr = (int)blockIdx.z, r = sh.row0 + lr;
  const int hp = (a.heads + 15) & ~15;                                         // heads in whole blocks; the rest weigh nothing
  float* s_m = reinterpret_cast<float*>(s_raw);                                // [hp]
  float* s_il = s_m + hp;                                                      // [hp]
  float* s_t = s_il + hp;                                                      // [hp][HG], T transposed
  float* s_w = s_t + hp * HG;                                                  // [32 warps][HG]
  float* s_red = s_w + blockDim.x * HG;                                       // [warps][HG][vpad]
  float* s_acc = s_red + (size_t)(blockDim.x >> 5) * HG * a.vpad;                      // [HG][vpad]
  int* s_row = reinterpret_cast<int*>(s_acc + HG * a.vpad);                    // [32 warps] cache rows
  const int vld = a.vpad + (VSM == 2 ? 8 : 0);
  T* s_v = reinterpret_cast<T*>(s_row + blockDim.x) + (size_t)(threadIdx.x >> 5) * 32 * vld;   // the warp's values when VSM
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nthr = (int)blockDim.x, nw = nthr >> 5;
  const int csize = (int)gridDim.x, crank = (int)blockIdx.x;   // CTAs that share the row's positions
  grid_dep_launch();
  for (int i = tid; i < hp * HG; i += nthr) {
    const int g = i / HG, h = i - g * HG;
    s_t[i] = h < nh && g < a.heads ? a.talk[(size_t)(h0 + h) * a.heads + g] : 0.f;
  }
  for (int i = lane; i < HG * a.vpad; i += 32) s_red[(size_t)warp * HG * a.vpad + i] = 0.f;
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first);
  const int nv = vr.count();
  const int64_t crow_elems = (int64_t)a.kv_heads * a.vpad;
  const T* vc = static_cast<const T*>(a.v_cache) + (pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows * crow_elems) + kv * a.vpad;
  // this CTA's positions, 32 per warp at a time
  const int v_begin = (int)((int64_t)nv * crank / csize), v_end = (int)((int64_t)nv * (crank + 1) / csize);
  auto stage = [&](int crow) {
    constexpr int EP = 16 / (int)sizeof(T);
    const int pieces = a.vpad / EP;
    int tr = lane / pieces, c = lane - tr * pieces;
    const int rstep = 32 / pieces, cstep = 32 - rstep * pieces;
    for (int i = 0; i < pieces; ++i) {
      const int src = __shfl_sync(0xffffffffu, crow, tr);
      cp16(s_v + tr * vld + c * EP, vc + (size_t)(uint32_t)src * (uint32_t)crow_elems + c * EP);
      tr += rstep;
      c += cstep;
      if (c >= pieces) { c -= pieces; ++tr; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (VSM && v_begin + warp * 32 < v_end) {   // the first values travel while the statistics are put together
    const int v = v_begin + warp * 32 + lane;
    stage(a.geom.row_of(vr.position(v < v_end ? v : v_begin + warp * 32)));
  }
  constexpr int GB = 16;                      // heads whose scores are requested together
  float pre[GB];                              // the first ones of the first positions
  const float* score_row = a.scores + (size_t)lr * a.heads * sh.stride;
  {
    const int v = v_begin + warp * 32 + lane;
#pragma unroll
    for (int j = 0; j < GB; ++j) pre[j] = j < a.heads && v < v_end ? score_row[(size_t)j * sh.stride + v] : 0.f;
  }
  constexpr int SB = 4;                       // softmax statistics from the parts, in a fixed order; SB heads in flight
  for (int g0 = warp * SB; g0 < hp; g0 += nw * SB) {
    float2 p0[SB], p1[SB];
#pragma unroll
    for (int j = 0; j < SB; ++j) {
      const float2* p = reinterpret_cast<const float2*>(a.part) + ((size_t)lr * a.heads + g0 + j) * sh.splits;
      p0[j] = p1[j] = make_float2(-INFINITY, 0.f);
      if (g0 + j < a.heads && lane < sh.splits) p0[j] = p[lane];
      if (g0 + j < a.heads && lane + 32 < sh.splits) p1[j] = p[lane + 32];
    }
    float m[SB], l[SB];
#pragma unroll
    for (int j = 0; j < SB; ++j) m[j] = fmaxf(p0[j].x, p1[j].x);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int j = 0; j < SB; ++j) m[j] = fmaxf(m[j], __shfl_xor_sync(0xffffffffu, m[j], o));
#pragma unroll
    for (int j = 0; j < SB; ++j)
      l[j] = (p0[j].x == -INFINITY ? 0.f : p0[j].y * expf(p0[j].x - m[j])) + (p1[j].x == -INFINITY ? 0.f : p1[j].y * expf(p1[j].x - m[j]));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int j = 0; j < SB; ++j) l[j] += __shfl_xor_sync(0xffffffffu, l[j], o);
    if (lane == 0)
#pragma unroll
      for (int j = 0; j < SB; ++j)
        if (g0 + j < hp) {
          // bf16: exp(s - m) / l as one exponential, 2^(s log2 e - (m log2 e + log2 l)).  A head that is only padding,
          // or a row that sees nothing: exp(-inf)
          s_m[g0 + j] = l[j] > 0.f ? (BF16 ? fmaf(m[j], kLog2E, log2f(l[j])) : m[j]) : INFINITY;
          s_il[g0 + j] = l[j] > 0.f ? 1.0f / l[j] : 0.f;
        }
  }
  __syncthreads();
  float* w_w = s_w + warp * 32 * HG;
  int* w_row = s_row + warp * 32;
  float* red = s_red + (size_t)warp * HG * a.vpad;
  constexpr int NT = VSM == 2 ? 16 : 1;       // 8-column tiles
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i] = 0.f;
  for (int v0 = v_begin + warp * 32; v0 < v_end; v0 += nthr) {
    const int v = v0 + lane;
    const bool live = v < v_end;
    const int crow = a.geom.row_of(vr.position(live ? v : v0));
    if (VSM) {
      if (v0 != v_begin + warp * 32) stage(crow);
    } else {
      w_row[lane] = crow;
    }
    const float* sp = score_row + (live ? v : v0);
    const bool first = v0 == v_begin + warp * 32;
    float w[HG];
#pragma unroll
    for (int h = 0; h < HG; ++h) w[h] = 0.f;
    for (int g0 = 0; g0 < a.heads; g0 += GB) {
      float s8[GB];
#pragma unroll
      for (int j = 0; j < GB; ++j, sp += sh.stride) s8[j] = first && g0 == 0 ? pre[j] : (g0 + j < a.heads ? *sp : 0.f);
#pragma unroll
      for (int j = 0; j < GB; ++j) {
        const int g = g0 + j;
        const float p = BF16 ? exp2f(fmaf(s8[j], kLog2E, -s_m[g])) : expf(s8[j] - s_m[g]) * s_il[g];
        float t[HG];
        load_row<HG>(s_t + g * HG, t);
#pragma unroll
        for (int h = 0; h < HG; ++h) w[h] = fmaf(t[h], p, w[h]);
      }
    }
#pragma unroll
    for (int h = 0; h < HG; ++h) w_w[lane * HG + h] = w[h];
    if (VSM) asm volatile("cp.async.wait_all;" ::: "memory");
    __syncwarp();
    const int nj = min(32, v_end - v0);
    if constexpr (VSM == 2) {
      // rows 0-3 of A: the weights of the heads rounded to bf16, rows 4-7: what the rounding left
      const int hr = (lane >> 2) & 3;
      const bool rest = lane >= 16;
#pragma unroll
      for (int kk = 0; kk < 32; kk += 16) {
        uint32_t wa[4] = {0u, 0u, 0u, 0u};
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int key = kk + x * 8 + (lane & 3) * 2;
          const float w0 = hr < HG && key < nj ? w_w[key * HG + hr] : 0.f, w1 = hr < HG && key + 1 < nj ? w_w[(key + 1) * HG + hr] : 0.f;
          const __nv_bfloat162 hi = __floats2bfloat162_rn(w0, w1);
          const float2 hf = __bfloat1622float2(hi);
          const __nv_bfloat162 lo = __floats2bfloat162_rn(w0 - hf.x, w1 - hf.y);
          wa[2 * x] = rest ? *reinterpret_cast<const uint32_t*>(&lo) : *reinterpret_cast<const uint32_t*>(&hi);
        }
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          if (n * 8 >= a.vpad) break;
          uint32_t vb[4];
          ldm4t(vb, s_v + (kk + (lane & 15)) * vld + n * 8 + (lane >> 4) * 8);
          mma16816(acc[n], wa, vb[0], vb[1]);
          mma16816(acc[n + 1 < NT ? n + 1 : n], wa, vb[2], vb[3]);
        }
      }
    } else if (VSM) {
      if (a.vpad > 64) warp_values<T, HG, 4>(s_v, nullptr, a.vpad, w_w, nj, a.vpad, red);
      else warp_values<T, HG, 2>(s_v, nullptr, a.vpad, w_w, nj, a.vpad, red);
    } else {
      warp_values<T, HG, 2>(vc, w_row, crow_elems, w_w, nj, a.vpad, red);
    }
    __syncwarp();
  }
  if constexpr (VSM == 2) {   // the two pieces' sums, into the warp's row sums
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float v = acc[n][i] + __shfl_xor_sync(0xffffffffu, acc[n][i], 16);
        if (lane < 16 && (lane >> 2) < HG && n * 8 < a.vpad) red[(lane >> 2) * a.vpad + n * 8 + (lane & 3) * 2 + i] = v;
      }
  }
  __syncthreads();
  for (int i = tid; i < HG * a.vpad; i += nthr) {
    float v = 0.f;
#pragma unroll 4
    for (int q = 0; q < nw; ++q) v += s_red[(size_t)q * HG * a.vpad + i];
    s_acc[i] = v;
  }
  __syncthreads();
  const int total = nh * a.vdim;
  for (int i = tid; i < total; i += nthr) {
    const int h = i / a.vdim, c = i - h * a.vdim;
    const float v = pos < 0 ? 0.f : s_acc[h * a.vpad + c];
    const int k = (h0 + h) * a.vdim + c;
    if (csize > 1) a.parts[((size_t)crank * sh.rows + lr) * ((size_t)a.heads * a.vdim) + k] = v;
    else act_store1<BF16>(a.out, r, k, v);
  }
  if (csize == 1 && h0 + nh == a.heads)
    for (int k = a.heads * a.vdim + tid; k < a.out.kp; k += nthr) act_store1<BF16>(a.out, r, k, 0.f);
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
    return ((query_bytes<T>(gq, a.dpad) + (size_t)w * gq * 8 + 15) & ~(size_t)15) + (size_t)w * kTileP * (a.dpad + 16 / sizeof(T)) * sizeof(T);
  };
  int warps = 8;
  while (warps > 1 && (sbytes(warps) > 112 * 1024 || warps / 2 >= tiles)) warps /= 2;
  int64_t splits = (2 * sm_count() + rows * a.kv_heads - 1) / (rows * a.kv_heads);
  if (splits > (tiles + warps - 1) / warps) splits = (tiles + warps - 1) / warps;
  if (splits > kScoreSplitsMax) splits = kScoreSplitsMax;
  sh.splits = (int)splits;
  // mix: query heads of one kv head per CTA; up to two CTAs per SM share a row's positions
  const int hg = gq >= 4 ? 4 : (gq >= 2 ? 2 : 1);
  const int groups = a.kv_heads * ((gq + hg - 1) / hg);
  int64_t mix_splits = 2 * sm_count() / (rows * groups);
  if (mix_splits > (a.max_visible + kMixThreads - 1) / kMixThreads) mix_splits = (a.max_visible + kMixThreads - 1) / kMixThreads;
  if (mix_splits > a.parts_rows / rows) mix_splits = a.parts_rows / rows;
  if (mix_splits < 1) mix_splits = 1;
  const size_t hp = ((size_t)a.heads + 15) & ~(size_t)15;
  size_t msm = 4 * (hp * (2 + hg) + (size_t)kMixThreads * hg + (size_t)(kMixThreads / 32 + 1) * hg * a.vpad + kMixThreads);
  const bool tensor = sizeof(T) == 2 && a.vpad <= 128;
  const size_t vsm = (size_t)kMixThreads * (a.vpad + (tensor ? 8 : 0)) * sizeof(T);
  const bool staged = msm + vsm <= 220 * 1024;
  if (staged) msm += vsm;
  if (sbytes(warps) > 200 * 1024 || msm > 220 * 1024)
    return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: attention with %d heads of size %d/%d", a.heads, a.dim, a.vdim);
  void (*mix)(WindowAttnArgs, ScoreShape) =
      staged ? (hg == 4 ? window_mix_kernel<T, BF16, 4, 1> : (hg == 2 ? window_mix_kernel<T, BF16, 2, 1> : window_mix_kernel<T, BF16, 1, 1>))
             : (hg == 4 ? window_mix_kernel<T, BF16, 4, 0> : (hg == 2 ? window_mix_kernel<T, BF16, 2, 0> : window_mix_kernel<T, BF16, 1, 0>));
  if constexpr (sizeof(T) == 2)
    if (staged && tensor) mix = hg == 4 ? window_mix_kernel<T, BF16, 4, 2> : (hg == 2 ? window_mix_kernel<T, BF16, 2, 2> : window_mix_kernel<T, BF16, 1, 2>);
  for (int64_t r0 = 0; r0 < a.r.rows; r0 += pass) {
    const int n = (int)(a.r.rows - r0 < pass ? a.r.rows - r0 : pass);
    sh.row0 = (int)r0;
    sh.rows = n;
    TB_TRY(launch_kernel(window_scores_kernel<T>, dim3((unsigned)sh.splits, (unsigned)a.kv_heads, (unsigned)n), dim3((unsigned)warps * 32),
                         sbytes(warps), st, a.pdl, 1, a, sh));
    TB_TRY(launch_kernel(mix, dim3((unsigned)mix_splits, (unsigned)groups, (unsigned)n), dim3(kMixThreads), msm, st, a.pdl, 1, a, sh));
    *launches += 2;
    if (mix_splits > 1) {
      TB_TRY(launch_window_parts(BF16 ? Precision::kBf16 : Precision::kF32, a, (int)mix_splits, (int)r0, n, st));
      ++*launches;
    }
  }
  return TB_OK;
}

// Sums over the splits of a row's positions, in order, as the next projection's operand.  grid (rows, columns / 256)
template <bool BF16>
__global__ void __launch_bounds__(256) window_parts_kernel(const WindowAttnArgs a, const int splits, const int row0, const int rows) {
  grid_dep_launch();
  grid_dep_wait();
  const int q = (int)blockIdx.x, k = (int)blockIdx.y * 256 + threadIdx.x, cols = a.heads * a.vdim;
  if (k >= a.out.kp) return;
  float v = 0.f;
  if (k < cols) {
#pragma unroll 8
    for (int z = 0; z < splits; ++z) v += a.parts[((size_t)z * rows + q) * cols + k];
  }
  act_store1<BF16>(a.out, row0 + q, k, v);
}

}  // namespace

tb_status launch_window_parts(Precision p, const WindowAttnArgs& a, int splits, int row0, int rows, cudaStream_t st) {
  const dim3 grid((unsigned)rows, (unsigned)((a.out.kp + 255) / 256));
  return p == Precision::kBf16 ? launch_kernel(window_parts_kernel<true>, grid, dim3(256), 0, st, a.pdl, 1, a, splits, row0, rows)
                               : launch_kernel(window_parts_kernel<false>, grid, dim3(256), 0, st, a.pdl, 1, a, splits, row0, rows);
}

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

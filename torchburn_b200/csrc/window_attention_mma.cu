// Windowed attention with mixed heads for a portion of one sequence in bf16: the two steps of
// window_attention.cu on the tensor cores.
//
//   scores   64 queries x one head per CTA: S = scale * Q K^T (mma.sync bf16, fp32 sums), masked, to scratch,
//            with each row's running maximum and sum
//   mix      16 queries x a group of heads per CTA, 32 keys at a time.  Mixing contracts over ALL heads at one
//            (query, key), so a thread owns two (query, key) pairs: it walks over the heads g, takes
//            exp(S - max) / sum once and adds T[h, g] times it to the group's weights, in registers, fp32.
//            The mixed weights go to shared memory as two bf16 pieces (together 16 mantissa bits; the second
//            piece is the rounding error of the first) and meet the values in two mma.sync each.
//
// Keys are numbered by the visible positions of the 64-query block: the kept positions, then one run from the
// first query's window to the last query.
#include "dense.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

constexpr int kQB = 64;      // queries per scores CTA; they share a key numbering
constexpr int kKeys = 64;    // keys per tile of the scores kernel
constexpr int kQM = 16;      // queries per mix CTA
constexpr int kKT = 32;      // keys per tile of the mix kernel
constexpr int kUnits = 8;    // 16-column output units per warp of the mix kernel
constexpr int kWStride = kKT + 8;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16z(void* dst, const void* src, bool live) {   // zeros when not live
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// The block's keys.  pos0: position of the block's first query, last: of its last one.
struct BlockKeys {
  int pos0, lo, nk, count;
  __device__ BlockKeys(int p0, int last, int window, int keep_first) : pos0(p0) {
    const VisibleRange a(p0, window, keep_first);
    lo = a.lo;
    nk = a.nk;
    count = nk + last - lo + 1;
  }
  __device__ int position(int v) const { return v < nk ? v : v - nk + lo; }
};

struct MmaShape {
  int64_t stride;   // floats per (row, head) of the score scratch
  int row0, rows;   // rows of this pass
};

// grid (heads, blocks of 64 queries), 128 threads
__global__ void __launch_bounds__(128) window_scores_mma_kernel(const WindowAttnArgs a, const MmaShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int ld = a.dpad + 8;   // row stride in elements: 16 bytes past a multiple of 32 bytes
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(s_raw);
  __nv_bfloat16* s_k = s_q + kQB * ld;             // two tiles
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = (int)blockIdx.x, kv = h / (a.heads / a.kv_heads);
  const int b0 = (int)blockIdx.y * kQB;            // first row of the block within the pass
  const int nrows = min(kQB, sh.rows - b0);
  grid_dep_launch();
  grid_dep_wait();
  const int r0 = sh.row0 + b0;
  const int pos0 = a.r.pos[r0];
  const BlockKeys keys(pos0, pos0 + nrows - 1, a.window, a.keep_first);
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.k_cache) + (size_t)a.r.slots[r0] * a.geom.rows * (size_t)(a.kv_heads * a.dpad) + (size_t)kv * a.dpad;
  const int pieces = a.dpad >> 3;
  for (int i = tid; i < kQB * pieces; i += 128) {
    const int r = i / pieces, c = i - r * pieces;
    const bool live = r < nrows;
    cp16z(s_q + r * ld + c * 8, a.q16 + ((size_t)(r0 + (live ? r : 0)) * a.heads + h) * a.dpad + c * 8, live);
  }
  auto fetch = [&](int t) {
    __nv_bfloat16* dst = s_k + (t & 1) * kKeys * ld;
    for (int i = tid; i < kKeys * pieces; i += 128) {
      const int r = i / pieces, c = i - r * pieces;
      const int v = t * kKeys + r;
      const bool live = v < keys.count;
      cp16z(dst + r * ld + c * 8, kc + (size_t)a.geom.row_of(keys.position(live ? v : 0)) * (a.kv_heads * a.dpad) + c * 8, live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int tiles = (keys.count + kKeys - 1) / kKeys;
  fetch(0);
  // the warp's 16 queries: this thread holds rows lane / 4 and lane / 4 + 8, key columns 2 (lane & 3) and the next
  const int qr[2] = {warp * 16 + (lane >> 2), warp * 16 + (lane >> 2) + 8};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  for (int t = 0; t < tiles; ++t) {
    if (t + 1 < tiles) {
      fetch(t + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const __nv_bfloat16* k = s_k + (t & 1) * kKeys * ld;
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
    for (int c = 0; c < a.dpad; c += 16) {
      uint32_t qa[4];
      ldm4(qa, s_q + (warp * 16 + (lane & 15)) * ld + c + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < 4; ++j) {   // 16 keys: matrices (keys 0-7, k 0-7) (keys 0-7, k 8-15) (keys 8-15, ...) ...
        uint32_t kb[4];
        ldm4(kb, k + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * ld + c + ((lane >> 3) & 1) * 8);
        mma16816(acc[2 * j], qa, kb[0], kb[1]);
        mma16816(acc[2 * j + 1], qa, kb[2], kb[3]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int pos = pos0 + qr[e];
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int v = t * kKeys + j * 8 + (lane & 3) * 2 + i;
          const int p = keys.position(v);
          const bool seen = v < keys.count && qr[e] < nrows && p <= pos && (pos - p < a.window || p < a.keep_first);
          const float s = seen ? acc[j][2 * e + i] * a.scale : -INFINITY;
          acc[j][2 * e + i] = s;
          mx = fmaxf(mx, s);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m1 = fmaxf(m[e], mx);
      float sum = 0.f;
      if (m1 != -INFINITY) {
#pragma unroll
        for (int j = 0; j < 8; ++j) sum += expf(acc[j][2 * e] - m1) + expf(acc[j][2 * e + 1] - m1);
        l[e] = l[e] * expf(m[e] - m1) + sum;
        m[e] = m1;
      }
      if (qr[e] < nrows) {
        float* dst = a.scores + ((size_t)(b0 + qr[e]) * a.heads + h) * sh.stride + t * kKeys + (lane & 3) * 2;
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (t * kKeys + j * 8 < keys.count) *reinterpret_cast<float2*>(dst + j * 8) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    if ((lane & 3) == 0 && qr[e] < nrows) {
      float* p = a.part + ((size_t)(b0 + qr[e]) * a.heads + h) * 2;
      p[0] = m[e];
      p[1] = l[e];
    }
  }
}

// grid (head groups, blocks of 16 queries), 256 threads.  HG: heads of a group (the last may be partly empty).
template <int HG>
__global__ void __launch_bounds__(256, 2) window_mix_mma_kernel(const WindowAttnArgs a, const MmaShape sh, const int kvs) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads;
  const int h0 = (int)blockIdx.x * HG, nh = min(HG, a.heads - h0);
  const int kv0 = h0 / gq, nkv = (h0 + nh - 1) / gq - kv0 + 1;
  const int vld = kvs * a.vpad + 8;
  float* s_t = reinterpret_cast<float*>(s_raw);                                   // [heads][HG], T transposed
  float2* s_ml = reinterpret_cast<float2*>(s_t + a.heads * HG);                   // [heads][kQM] (max, 1 / sum)
  __nv_bfloat16* s_w = reinterpret_cast<__nv_bfloat16*>(s_ml + a.heads * kQM);    // [HG][2 pieces][kQM][kWStride]
  __nv_bfloat16* s_v = s_w + HG * 2 * kQM * kWStride;                             // [kKT][vld]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int q0 = (int)blockIdx.y * kQM;              // first row within the pass
  const int nrows = min(kQM, sh.rows - q0);
  const int b0 = q0 / kQB * kQB;
  grid_dep_launch();
  grid_dep_wait();
  const int pos_b = a.r.pos[sh.row0 + b0];
  const BlockKeys keys(pos_b, pos_b + min(kQB, sh.rows - b0) - 1, a.window, a.keep_first);
  const int pos0 = pos_b + q0 - b0, pos1 = pos0 + nrows - 1;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v_cache) + (size_t)a.r.slots[sh.row0] * a.geom.rows * (size_t)(a.kv_heads * a.vpad) + (size_t)kv0 * a.vpad;
  for (int i = tid; i < a.heads * HG; i += 256) {
    const int g = i / HG, h = i - g * HG;
    s_t[i] = h < nh ? a.talk[(size_t)(h0 + h) * a.heads + g] : 0.f;
  }
  for (int i = tid; i < a.heads * kQM; i += 256) {
    const int g = i / kQM, q = i - g * kQM;
    float2 v = make_float2(0.f, 0.f);
    if (q < nrows) {
      const float* p = a.part + ((size_t)(q0 + q) * a.heads + g) * 2;
      v = make_float2(p[0], p[1] > 0.f ? 1.0f / p[1] : 0.f);
    }
    s_ml[i] = v;
  }
  // tiles that hold a key one of these queries sees
  const VisibleRange first(pos0, a.window, a.keep_first);
  const int kept_tiles = (min(a.keep_first, keys.count) + kKT - 1) / kKT;   // a kept position's number is the position itself
  const int win0 = (keys.nk + first.lo - keys.lo) / kKT, win1 = (keys.nk + pos1 - keys.lo) / kKT;
  const int pieces = nkv * a.vpad >> 3;
  const int upv = a.vpad >> 4, units = nh * upv;     // 16-column output units
  float acc[kUnits][2][4];
#pragma unroll
  for (int u = 0; u < kUnits; ++u)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[u][j][i] = 0.f;
  for (int t = 0; t <= win1; ++t) {
    if (t >= kept_tiles && t < win0) { t = win0 - 1; continue; }
    __syncthreads();
    for (int i = tid; i < kKT * pieces; i += 256) {
      const int r = i / pieces, c = i - r * pieces;
      const int v = t * kKT + r;
      const bool live = v < keys.count;
      cp16z(s_v + r * vld + c * 8, vc + (size_t)a.geom.row_of(keys.position(live ? v : 0)) * (a.kv_heads * a.vpad) + c * 8, live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    // mixed weights of (query warp, key lane) and (query warp + 8, key lane)
    float w[2][HG];
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int h = 0; h < HG; ++h) w[e][h] = 0.f;
    const int v = t * kKT + lane;
    const bool in0 = v < keys.count && warp < nrows, in1 = v < keys.count && warp + 8 < nrows;
    const float* sp0 = a.scores + (size_t)(q0 + (in0 ? warp : 0)) * a.heads * sh.stride + (in0 ? v : 0);
    const float* sp1 = a.scores + (size_t)(q0 + (in1 ? warp + 8 : 0)) * a.heads * sh.stride + (in1 ? v : 0);
    constexpr int GB = 4;                            // heads whose scores are requested together
    for (int g0 = 0; g0 < a.heads; g0 += GB) {
      float s0[GB], s1[GB];
#pragma unroll
      for (int j = 0; j < GB; ++j) {
        const bool lg = g0 + j < a.heads;
        s0[j] = in0 && lg ? __ldg(sp0 + (size_t)(g0 + j) * sh.stride) : -INFINITY;
        s1[j] = in1 && lg ? __ldg(sp1 + (size_t)(g0 + j) * sh.stride) : -INFINITY;
      }
#pragma unroll
      for (int j = 0; j < GB; ++j) {
        if (g0 + j >= a.heads) break;
        const float2 ml0 = s_ml[(g0 + j) * kQM + warp], ml1 = s_ml[(g0 + j) * kQM + warp + 8];
        const float p0 = expf(s0[j] - ml0.x) * ml0.y, p1 = expf(s1[j] - ml1.x) * ml1.y;
        const float* tr = s_t + (g0 + j) * HG;
#pragma unroll
        for (int h = 0; h < HG; h += 4) {
          const float4 tv = *reinterpret_cast<const float4*>(tr + h);
          w[0][h] = fmaf(tv.x, p0, w[0][h]); w[0][h + 1] = fmaf(tv.y, p0, w[0][h + 1]);
          w[0][h + 2] = fmaf(tv.z, p0, w[0][h + 2]); w[0][h + 3] = fmaf(tv.w, p0, w[0][h + 3]);
          w[1][h] = fmaf(tv.x, p1, w[1][h]); w[1][h + 1] = fmaf(tv.y, p1, w[1][h + 1]);
          w[1][h + 2] = fmaf(tv.z, p1, w[1][h + 2]); w[1][h + 3] = fmaf(tv.w, p1, w[1][h + 3]);
        }
      }
    }
#pragma unroll
    for (int h = 0; h < HG; ++h)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const __nv_bfloat16 hi = __float2bfloat16_rn(w[e][h]);
        __nv_bfloat16* d = s_w + (size_t)(h * 2) * kQM * kWStride + (warp + 8 * e) * kWStride + lane;
        d[0] = hi;
        d[kQM * kWStride] = __float2bfloat16_rn(w[e][h] - __bfloat162float(hi));
      }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
#pragma unroll
    for (int u = 0; u < kUnits; ++u) {
      const int unit = warp + 8 * u;
      if (unit >= units) break;
      const int h = unit / upv, c = (unit - h * upv) * 16;
      const __nv_bfloat16* wp = s_w + (size_t)(h * 2) * kQM * kWStride;
      const __nv_bfloat16* vp = s_v + ((h0 + h) / gq - kv0) * a.vpad + c;
#pragma unroll
      for (int kk = 0; kk < kKT; kk += 16) {
        uint32_t hi[4], lo[4], vb[4];
        const int off = (lane & 15) * kWStride + kk + (lane >> 4) * 8;
        ldm4(hi, wp + off);
        ldm4(lo, wp + kQM * kWStride + off);
        // V is [key][column]: transposed loads give (keys 0-7, cols 0-7) (keys 8-15, cols 0-7) (keys 0-7, cols 8-15) ...
        ldm4t(vb, vp + (kk + (lane & 15)) * vld + (lane >> 4) * 8);
        mma16816(acc[u][0], hi, vb[0], vb[1]);
        mma16816(acc[u][1], hi, vb[2], vb[3]);
        mma16816(acc[u][0], lo, vb[0], vb[1]);
        mma16816(acc[u][1], lo, vb[2], vb[3]);
      }
    }
  }
#pragma unroll
  for (int u = 0; u < kUnits; ++u) {
    const int unit = warp + 8 * u;
    if (unit >= units) break;
    const int h = unit / upv, c = (unit - h * upv) * 16;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int q = (lane >> 2) + (i >> 1) * 8, col = c + j * 8 + (lane & 3) * 2 + (i & 1);
        if (q < nrows && col < a.vdim) act_store1<true>(a.out, sh.row0 + q0 + q, (h0 + h) * a.vdim + col, acc[u][j][i]);
      }
  }
  if (h0 + nh == a.heads)
    for (int q = 0; q < nrows; ++q)
      for (int k = a.heads * a.vdim + tid; k < a.out.kp; k += 256) act_store1<true>(a.out, sh.row0 + q0 + q, k, 0.f);
}

size_t mix_bytes(const WindowAttnArgs& a, int hg, int kvs) {
  return (size_t)a.heads * hg * 4 + (size_t)a.heads * kQM * 8 + (size_t)hg * 2 * kQM * kWStride * 2 + (size_t)kKT * (kvs * a.vpad + 8) * 2;
}

}  // namespace

bool window_mma_supported(const WindowAttnArgs& a) {
  return a.one_sequence && a.q16 != nullptr && a.r.rows >= kQM && a.dpad <= 256 && a.vpad <= 256 && a.heads <= 128;
}

tb_status launch_window_attention_mma(const WindowAttnArgs& a, cudaStream_t st, int* launches) {
  const int gq = a.heads / a.kv_heads;
  // heads per group: as many as the accumulators hold, fewer while the grid leaves SMs idle
  int hg = a.vpad <= 64 ? 16 : (a.vpad <= 128 ? 8 : 4);
  while (hg > 4 && (hg / 2 >= a.heads || (int64_t)((a.r.rows + kQM - 1) / kQM) * ((a.heads + hg - 1) / hg) < sm_count())) hg /= 2;
  int kvs = hg % gq == 0 ? hg / gq : (gq % hg == 0 ? 1 : (hg + gq - 2) / gq + 1);
  if (kvs > a.kv_heads) kvs = a.kv_heads;
  MmaShape sh;
  sh.stride = (int64_t)window_attn_score_stride(a.max_visible);
  int64_t pass = a.scratch_rows >= a.r.rows ? a.r.rows : a.scratch_rows / kQB * kQB;
  if (pass < 1) return fail(TB_ERR_UNSUPPORTED, "window attention: score scratch holds %lld rows", (long long)a.scratch_rows);
  const size_t ssm = (size_t)(kQB + 2 * kKeys) * (a.dpad + 8) * 2, msm = mix_bytes(a, hg, kvs);
  for (int64_t r0 = 0; r0 < a.r.rows; r0 += pass) {
    sh.row0 = (int)r0;
    sh.rows = (int)(a.r.rows - r0 < pass ? a.r.rows - r0 : pass);
    TB_TRY(launch_kernel(window_scores_mma_kernel, dim3((unsigned)a.heads, (unsigned)((sh.rows + kQB - 1) / kQB)), dim3(128), ssm, st, a.pdl, 1, a, sh));
    const dim3 grid((unsigned)((a.heads + hg - 1) / hg), (unsigned)((sh.rows + kQM - 1) / kQM));
    auto* kern = hg == 16 ? window_mix_mma_kernel<16> : (hg == 8 ? window_mix_mma_kernel<8> : window_mix_mma_kernel<4>);
    TB_TRY(launch_kernel(kern, grid, dim3(256), msm, st, a.pdl, 1, a, sh, kvs));
    *launches += 2;
  }
  return TB_OK;
}

}  // namespace tb

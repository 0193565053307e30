// Windowed attention with mixed heads for a portion of one sequence in bf16: the two steps of
// window_attention.cu on the tensor cores.
//
//   scores   64 queries x one head per CTA: S = scale * Q K^T (mma.sync bf16, fp32 sums), masked, to scratch,
//            with each row's running maximum and sum
//   mix      16 queries x a group of up to 16 heads per CTA, 32 keys at a time.  weights = exp(S - max) / sum of
//            ALL heads at a (query, key) are contracted with T over the heads: one mma.sync per 16 x 16 heads
//            and 8 keys (T is exact in bf16; a weight goes in as two bf16 pieces, the second one the rounding
//            error of the first: 16 mantissa bits).  The mixed weights, again two pieces, meet the values in
//            two mma.sync each.  Scores and values of the next 32 keys stream in meanwhile.  With few query
//            blocks several CTAs share the keys of one; their parts are plain sums (the weights are normalised
//            already) and a last kernel adds them in order.
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
constexpr int kMixThreads = 512, kMixWarps = 16;
constexpr int kUnits = 8;      // 16-column output units per warp of the mix kernel
constexpr int kWStride = kKT + 8;
constexpr int kWHead = 2 * kQM * kWStride + 32;   // elements of one head's two pieces
constexpr int kSStride = kKT + 4;                 // floats per (query, head) row of staged scores
constexpr int kMaxKeySplits = 4;

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

struct MmaShape {
  int64_t stride;   // floats per (row, head) of the score scratch
  int row0, rows;   // rows of this pass
  int hg, kvs;      // mix: heads per group, most kv heads a group touches
  int score_splits; // scores: CTAs that share a query block's keys
  int key_splits;   // mix: CTAs that share a query block's keys
};

// grid (heads, blocks of 64 queries, score splits), 128 threads
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
  int lsh = 1;                                     // 2^lsh threads per row
  while ((1 << lsh) < pieces) ++lsh;
  const int c0 = tid & ((1 << lsh) - 1), rr0 = tid >> lsh, rstep = 128 >> lsh;
  if (c0 < pieces)
    for (int r = rr0; r < kQB; r += rstep) {
      const bool live = r < nrows;
      cp16z(s_q + r * ld + c0 * 8, a.q16 + ((size_t)(r0 + (live ? r : 0)) * a.heads + h) * a.dpad + c0 * 8, live);
    }
  const int krow = a.kv_heads * a.dpad;
  auto fetch = [&](int t) {
    __nv_bfloat16* dst = s_k + (t & 1) * kKeys * ld;
    const RunRows rows(keys, a.geom, t * kKeys);
    if (c0 < pieces)
      for (int r = rr0; r < kKeys; r += rstep) {
        const int v = t * kKeys + r;
        const bool live = v < keys.count;
        cp16z(dst + r * ld + c0 * 8, kc + (size_t)(live ? rows.row(v) : 0) * krow + c0 * 8, live);
      }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int tiles = (keys.count + kKeys - 1) / kKeys;
  const int t0 = (int)((int64_t)tiles * blockIdx.z / sh.score_splits), t1 = (int)((int64_t)tiles * (blockIdx.z + 1) / sh.score_splits);
  if (t0 < t1) fetch(t0);
  // the warp's 16 queries: this thread holds rows lane / 4 and lane / 4 + 8, key columns 2 (lane & 3) and the next
  const int qr[2] = {warp * 16 + (lane >> 2), warp * 16 + (lane >> 2) + 8};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  for (int t = t0; t < t1; ++t) {
    if (t + 1 < t1) {
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
    // every key of the tile seen by every query of the block?
    const int vf = t * kKeys;
    const bool all_seen = nrows == kQB && vf >= keys.nk && vf + kKeys <= keys.count && keys.position(vf + kKeys - 1) <= pos0 &&
                          pos0 + kQB - 1 - keys.position(vf) < a.window;
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
          const bool seen = all_seen || (v < keys.count && qr[e] < nrows && p <= pos && (pos - p < a.window || p < a.keep_first));
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
      float* p = a.part + (((size_t)(b0 + qr[e]) * a.heads + h) * sh.score_splits + blockIdx.z) * 2;
      p[0] = m[e];
      p[1] = l[e];
    }
  }
}

// grid (head groups, blocks of 16 queries, key splits)
template <bool STAGED>
__global__ void __launch_bounds__(kMixThreads, 1) window_mix_mma_kernel(const WindowAttnArgs a, const MmaShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  const int gq = a.heads / a.kv_heads, hp = (a.heads + 15) & ~15;
  const int h0 = (int)blockIdx.x * sh.hg, nh = min(sh.hg, a.heads - h0);
  const int kv0 = h0 / gq, nkv = (h0 + nh - 1) / gq - kv0 + 1;
  const int vld = sh.kvs * a.vpad + 8, tld = hp + 8;
  float2* s_ml = reinterpret_cast<float2*>(s_raw);                                // [hp][kQM] (max, 1 / sum)
  __nv_bfloat16* s_t = reinterpret_cast<__nv_bfloat16*>(s_ml + hp * kQM);         // [16][tld] rows of T
  __nv_bfloat16* s_w = s_t + 16 * tld;                                            // [hg][kWHead]
  __nv_bfloat16* s_v = s_w + sh.hg * kWHead;                                      // [2][kKT][vld]
  float* s_s = reinterpret_cast<float*>(s_v + 2 * kKT * vld);                     // [kQM][heads][kSStride] when STAGED
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int q0 = (int)blockIdx.y * kQM;              // first row within the pass
  const int nrows = min(kQM, sh.rows - q0);
  const int b0 = q0 / kQB * kQB;
  grid_dep_launch();
  for (int i = tid; i < 16 * hp; i += kMixThreads) {
    const int h = i / hp, g = i - h * hp;
    s_t[h * tld + g] = __float2bfloat16_rn(h < nh && g < a.heads ? a.talk[(size_t)(h0 + h) * a.heads + g] : 0.f);
  }
  grid_dep_wait();
  const int pos_b = a.r.pos[sh.row0 + b0];
  const BlockKeys keys(pos_b, pos_b + min(kQB, sh.rows - b0) - 1, a.window, a.keep_first);
  const int pos0 = pos_b + q0 - b0, pos1 = pos0 + nrows - 1;
  const int vrow = a.kv_heads * a.vpad;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v_cache) + (size_t)a.r.slots[sh.row0] * a.geom.rows * (size_t)vrow + (size_t)kv0 * a.vpad;
  for (int i = tid; i < hp * kQM; i += kMixThreads) {
    const int g = i / kQM, q = i - g * kQM;
    float2 v = make_float2(INFINITY, 0.f);           // a dead row's weights are exp(-inf) = 0
    if (q < nrows && g < a.heads) {
      const float* p = a.part + ((size_t)(q0 + q) * a.heads + g) * sh.score_splits * 2;
      float m = p[0], l = p[1];
      for (int z = 1; z < sh.score_splits; ++z) {      // in order
        const float m2 = p[2 * z], l2 = p[2 * z + 1], m1 = fmaxf(m, m2);
        l = (m == -INFINITY ? 0.f : l * expf(m - m1)) + (m2 == -INFINITY ? 0.f : l2 * expf(m2 - m1));
        m = m1;
      }
      v = make_float2(m, 1.0f / l);
    }
    s_ml[i] = v;
  }
  // tiles that hold a key one of these queries sees: the kept positions (their numbers are the positions), the run
  const VisibleRange first(pos0, a.window, a.keep_first);
  const int win1 = (keys.nk + pos1 - keys.lo) / kKT;
  const int kept = min((min(a.keep_first, keys.count) + kKT - 1) / kKT, win1 + 1);
  const int win0 = max(kept, (keys.nk + first.lo - keys.lo) / kKT);
  const int total = kept + win1 + 1 - win0;
  const int n0 = (int)((int64_t)total * blockIdx.z / sh.key_splits), n1 = (int)((int64_t)total * (blockIdx.z + 1) / sh.key_splits);
  const int pieces = nkv * a.vpad >> 3;
  auto fetch = [&](int n) {
    const int t = n < kept ? n : win0 + n - kept;
    __nv_bfloat16* dst = s_v + (n & 1) * kKT * vld;
    const RunRows rows(keys, a.geom, t * kKT);
    for (int r = warp; r < kKT; r += kMixWarps) {
      const int v = t * kKT + r;
      const bool live = v < keys.count;
      const __nv_bfloat16* src = vc + (size_t)(live ? rows.row(v) : 0) * vrow;
      for (int c = lane; c < pieces; c += 32) cp16z(dst + r * vld + c * 8, src + c * 8, live);
    }
    if (STAGED) {
      // warp = query, 4 heads x 8 pieces of 4 keys at a time
      const int q = warp < nrows ? warp : 0;
      const float* src = a.scores + (size_t)(q0 + q) * a.heads * sh.stride + t * kKT + (lane & 7) * 4;
      float* d = s_s + (size_t)warp * a.heads * kSStride + (lane & 7) * 4;
      for (int g = lane >> 3; g < a.heads; g += 4) cp16z(d + g * kSStride, src + (size_t)g * sh.stride, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int upv = a.vpad >> 4, units = nh * upv;     // 16-column output units
  float acc[kUnits][2][4];
#pragma unroll
  for (int u = 0; u < kUnits; ++u)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[u][j][i] = 0.f;
  if (n0 < n1) fetch(n0);
  for (int n = n0; n < n1; ++n) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    // ---- mixed weights of query `warp` at the tile's keys: lane / 4 = column n of the MMA = keys 4 n .. 4 n + 3 ----
    const int t = n < kept ? n : win0 + n - kept;
    const int kn = (lane >> 2) * 4, left = keys.count - (t * kKT + kn);   // keys of this thread that exist
    float d[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i) d[k][i] = 0.f;
    const float* sp = STAGED ? s_s + (size_t)warp * a.heads * kSStride + kn
                             : a.scores + (size_t)(q0 + (warp < nrows ? warp : 0)) * a.heads * sh.stride + t * kKT + kn;
    const int64_t gstride = STAGED ? kSStride : sh.stride;
    for (int kg = 0; kg < hp; kg += 16) {
      uint32_t ta[4];
      ldm4(ta, s_t + (lane & 15) * tld + kg + (lane >> 4) * 8);
      float p[4][4];                                   // [head of the fragment][key]
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int g = kg + (lane & 3) * 2 + (j & 1) + (j >> 1) * 8;
        float4 s4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (g < a.heads) s4 = *reinterpret_cast<const float4*>(sp + (size_t)g * gstride);
        const float2 ml = s_ml[g * kQM + warp];
        p[j][0] = left > 0 ? expf(s4.x - ml.x) * ml.y : 0.f;
        p[j][1] = left > 1 ? expf(s4.y - ml.x) * ml.y : 0.f;
        p[j][2] = left > 2 ? expf(s4.z - ml.x) * ml.y : 0.f;
        p[j][3] = left > 3 ? expf(s4.w - ml.x) * ml.y : 0.f;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t hi[2], lo[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const __nv_bfloat162 hv = __floats2bfloat162_rn(p[2 * j][k], p[2 * j + 1][k]);
          const float2 hf = __bfloat1622float2(hv);
          const __nv_bfloat162 lv = __floats2bfloat162_rn(p[2 * j][k] - hf.x, p[2 * j + 1][k] - hf.y);
          hi[j] = *reinterpret_cast<const uint32_t*>(&hv);
          lo[j] = *reinterpret_cast<const uint32_t*>(&lv);
        }
        mma16816(d[k], ta, hi[0], hi[1]);
        mma16816(d[k], ta, lo[0], lo[1]);
      }
    }
    // d[k][2 a + b]: head lane / 4 + 8 a, column 2 (lane & 3) + b, key k of the column
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int h = (lane >> 2) + (i >> 1) * 8, key = ((lane & 3) * 2 + (i & 1)) * 4;
      if (h < nh) {
        const __nv_bfloat162 h01 = __floats2bfloat162_rn(d[0][i], d[1][i]), h23 = __floats2bfloat162_rn(d[2][i], d[3][i]);
        const float2 f01 = __bfloat1622float2(h01), f23 = __bfloat1622float2(h23);
        const __nv_bfloat162 l01 = __floats2bfloat162_rn(d[0][i] - f01.x, d[1][i] - f01.y), l23 = __floats2bfloat162_rn(d[2][i] - f23.x, d[3][i] - f23.y);
        __nv_bfloat16* wp = s_w + (size_t)h * kWHead + warp * kWStride + key;
        *reinterpret_cast<uint2*>(wp) = make_uint2(*reinterpret_cast<const uint32_t*>(&h01), *reinterpret_cast<const uint32_t*>(&h23));
        *reinterpret_cast<uint2*>(wp + kQM * kWStride) = make_uint2(*reinterpret_cast<const uint32_t*>(&l01), *reinterpret_cast<const uint32_t*>(&l23));
      }
    }
    __syncthreads();
    if (n + 1 < n1) fetch(n + 1);
    const __nv_bfloat16* vt = s_v + (n & 1) * kKT * vld;
#pragma unroll
    for (int u = 0; u < kUnits; ++u) {
      const int unit = warp + kMixWarps * u;
      if (unit >= units) break;
      const int h = unit / upv, c = (unit - h * upv) * 16;
      const __nv_bfloat16* wp = s_w + (size_t)h * kWHead;
      const __nv_bfloat16* vp = vt + ((h0 + h) / gq - kv0) * a.vpad + c;
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
  const int cols = a.heads * a.vdim;
#pragma unroll
  for (int u = 0; u < kUnits; ++u) {
    const int unit = warp + kMixWarps * u;
    if (unit >= units) break;
    const int h = unit / upv, c = (unit - h * upv) * 16;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int q = (lane >> 2) + (i >> 1) * 8, col = c + j * 8 + (lane & 3) * 2 + (i & 1);
        if (q >= nrows || col >= a.vdim) continue;
        const int k = (h0 + h) * a.vdim + col;
        if (sh.key_splits > 1) a.parts[((size_t)blockIdx.z * sh.rows + q0 + q) * cols + k] = acc[u][j][i];
        else act_store1<true>(a.out, sh.row0 + q0 + q, k, acc[u][j][i]);
      }
  }
  if (sh.key_splits == 1 && h0 + nh == a.heads)
    for (int q = 0; q < nrows; ++q)
      for (int k = cols + tid; k < a.out.kp; k += kMixThreads) act_store1<true>(a.out, sh.row0 + q0 + q, k, 0.f);
}

size_t mix_bytes(const WindowAttnArgs& a, int hg, int kvs, bool staged) {
  const int hp = (a.heads + 15) & ~15;
  return (size_t)hp * kQM * 8 + (size_t)16 * (hp + 8) * 2 + (size_t)hg * kWHead * 2 + (size_t)2 * kKT * (kvs * a.vpad + 8) * 2 +
         (staged ? (size_t)kQM * a.heads * kSStride * 4 : 0);
}
int group_kv_heads(const WindowAttnArgs& a, int hg) {   // most kv heads a group of hg query heads touches
  const int gq = a.heads / a.kv_heads;
  const int n = hg % gq == 0 ? hg / gq : (gq % hg == 0 ? 1 : (hg + gq - 2) / gq + 1);
  return n < a.kv_heads ? n : a.kv_heads;
}
constexpr size_t kSmemMax = 226 * 1024;

}  // namespace

bool window_mma_supported(const WindowAttnArgs& a) {
  return a.one_sequence && a.q16 != nullptr && a.r.rows >= kQM && a.dpad <= 256 && a.vpad <= 256 && a.heads <= 256 && (a.scratch_rows >= kQB || a.scratch_rows >= a.r.rows) &&
         mix_bytes(a, 1, 1, false) <= kSmemMax;
}

tb_status launch_window_attention_mma(const WindowAttnArgs& a, cudaStream_t st, int* launches) {
  // heads per group: as many as one MMA holds and accumulators and shared memory allow
  int hg = 16;
  while (hg > 1 && (hg / 2 >= a.heads || hg * a.vpad > kUnits * kMixWarps * 16 || mix_bytes(a, hg, group_kv_heads(a, hg), false) > kSmemMax)) hg /= 2;
  MmaShape sh;
  sh.hg = hg;
  sh.kvs = group_kv_heads(a, hg);
  sh.stride = (int64_t)window_attn_score_stride(a.max_visible);
  const bool staged = mix_bytes(a, hg, sh.kvs, true) <= kSmemMax;
  // passes of equal size, in whole query blocks, as many rows as the score scratch holds
  const int64_t blocks = (a.r.rows + kQB - 1) / kQB, fit = a.scratch_rows / kQB;
  const int64_t passes = a.scratch_rows >= a.r.rows ? 1 : (blocks + fit - 1) / fit;
  const int64_t pass = (blocks + passes - 1) / passes * kQB;
  const int groups = (a.heads + hg - 1) / hg;
  const size_t ssm = (size_t)(kQB + 2 * kKeys) * (a.dpad + 8) * 2, msm = mix_bytes(a, hg, sh.kvs, staged);
  for (int64_t r0 = 0; r0 < a.r.rows; r0 += pass) {
    sh.row0 = (int)r0;
    sh.rows = (int)(a.r.rows - r0 < pass ? a.r.rows - r0 : pass);
    const int64_t qb = (sh.rows + kQB - 1) / kQB;
    sh.score_splits = 1;
    while (sh.score_splits < 8 && a.heads * qb * sh.score_splits < 4 * sm_count() && a.max_visible >= (int64_t)kKeys * 4 * sh.score_splits) sh.score_splits *= 2;
    TB_TRY(launch_kernel(window_scores_mma_kernel, dim3((unsigned)a.heads, (unsigned)qb, (unsigned)sh.score_splits), dim3(128), ssm, st, a.pdl, 1, a, sh));
    const int qblocks = (sh.rows + kQM - 1) / kQM;
    sh.key_splits = 1;
    while (sh.key_splits < kMaxKeySplits && a.parts_rows >= 2 * (int64_t)sh.rows * sh.key_splits && groups * qblocks * sh.key_splits * 3 / 2 < sm_count() &&
           a.max_visible >= (int64_t)kKT * 8 * sh.key_splits)
      sh.key_splits *= 2;
    auto* kern = staged ? window_mix_mma_kernel<true> : window_mix_mma_kernel<false>;
    TB_TRY(launch_kernel(kern, dim3((unsigned)groups, (unsigned)qblocks, (unsigned)sh.key_splits), dim3(kMixThreads), msm, st, a.pdl, 1, a, sh));
    *launches += 2;
    if (sh.key_splits > 1) {
      TB_TRY(launch_window_parts(Precision::kBf16, a, sh.key_splits, sh.row0, sh.rows, st));
      ++*launches;
    }
  }
  return TB_OK;
}

}  // namespace tb

// Attention with an online softmax: grouped heads, a window with kept first positions or chunks of the sequence, a
// soft cap on the scores, a distance bias per head, an output gate per head; or one latent shared by all heads, whose
// first elements are also the values.
//
//   score(i, j) = cap(scale q_i . k_j) - slope_h (i - j),   cap(s) = softcap tanh(s / softcap)
//
// bf16, decode steps with up to eight query heads per key head (flash_decode_kernel): a warp takes 32 keys at a time from
// their load to its own running output and needs no other warp until the end; keys are the 16-row side of mma.sync, the
// heads its eight columns.
// bf16 otherwise (flash_mma_kernel): a CTA takes up to 64 (query, head) pairs of one key/value head - the heads of one row in
// a decode step, several queries times the heads in a portion - so that heads that share keys share their loads.
// Per tile of 32 or 64 keys: scores by mma.sync with the warps side by side over the keys, softmax weights to shared
// memory as two bf16 pieces (the second one what the rounding of the first left: 16 mantissa bits), then the values
// with the warps side by side over the value columns.  CTAs that share a block's keys leave (max, sum, unnormalised
// output) and a last kernel merges them in a fixed order.
// Portions of one sequence take the tcgen05 kernel of flash_tc5.cu where its tiles fit, decode steps over latents that of
// flash_latent.cu.
// fp32, and sizes beyond the tiles (flash_simple_kernel): a CTA per row and up to four heads, fp32 products.
#include "dense.cuh"
#include "flash_attention.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

constexpr int kThreads = 256;
constexpr float kLog2E = 1.44269504f;
constexpr int kMaxSplits = 512;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16z(void* dst, const void* src, bool live) {   // zeros when not live
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldm2(uint32_t (&r)[2], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// First positions that a row sees in its own run.
__device__ __forceinline__ int run_start(const FlashArgs& a, int pos) { return VisibleRange(pos, a.window, 0, a.chunk).lo; }

// grid (tiles * splits, kv heads, runs)
template <int MG, int NV, int KT>
__global__ void __launch_bounds__(kThreads, NV <= 8 ? 2 : 1) flash_mma_kernel(const FlashArgs a, const FlashShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  constexpr int M = 16 * MG, WN = 8 / MG, KW = KT / WN, NS = KW / 8, PLD = KT + 8;
  static_assert(NS >= 1, "a warp takes at least eight keys");
  const int gq = a.heads / a.kv_heads, kv = (int)blockIdx.y;
  const int split = (int)blockIdx.x % sh.splits, tile = sh.tiles - 1 - (int)blockIdx.x / sh.splits;   // the longest tiles first
  const int row0 = (int)blockIdx.z * sh.run_rows, pairs = sh.run_rows * gq;
  const int p0 = tile * M, np = min(M, pairs - p0);
  const int ld = a.dpad + 8, vld = a.values_in_keys ? ld : a.vpad + 8;
  __nv_bfloat16* s_q = reinterpret_cast<__nv_bfloat16*>(s_raw);             // [M][ld]
  __nv_bfloat16* s_k = s_q + M * ld;                                        // [2][KT][ld]
  __nv_bfloat16* s_v = a.values_in_keys ? s_k : s_k + 2 * KT * ld;          // [2][KT][vld]
  __nv_bfloat16* s_p = a.values_in_keys ? s_k + 2 * KT * ld : s_v + 2 * KT * vld;   // [2 pieces][M][PLD]
  float* s_max = reinterpret_cast<float*>(s_p + 2 * M * PLD);               // [WN][M]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wr = warp % MG, wc = warp / MG;
  grid_dep_launch();
  grid_dep_wait();
  const int pos_r = a.r.pos[row0];
  const int first = pos_r + p0 / gq;
  int last = pos_r + (p0 + np - 1) / gq;
  if (a.geom.ring == 0) last = min(last, (int)a.geom.rows - 1);
  const BlockKeys keys(first, pos_r < 0 ? -1 : last, a.window, a.keep_first, a.chunk);
  const size_t slot = pos_r < 0 ? 0 : (size_t)a.r.slots[row0];
  const int krow = a.kv_heads * a.dpad, vrow = a.kv_heads * a.vpad;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.k_cache) + slot * a.geom.rows * (size_t)krow + (size_t)kv * a.dpad;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v_cache) + (a.values_in_keys ? 0 : slot * a.geom.rows * (size_t)vrow + (size_t)kv * a.vpad);
  // 2^lsh threads per row of 16-byte pieces
  auto log_threads = [](int pieces) {
    int l = 1;
    while ((1 << l) < pieces) ++l;
    return l;
  };
  const int kpieces = a.dpad >> 3, vpieces = a.vpad >> 3, klsh = log_threads(kpieces), vlsh = log_threads(vpieces);
  auto fetch = [&](int t) {
    const RunRows rows(keys, a.geom, t * KT);
    {
      const int c = tid & ((1 << klsh) - 1);
      __nv_bfloat16* dst = s_k + (t & 1) * KT * ld + c * 8;
      if (c < kpieces)
        for (int r = tid >> klsh; r < KT; r += kThreads >> klsh) {
          const int v = t * KT + r;
          const bool live = v < keys.count;
          cp16z(dst + r * ld, kc + (size_t)(live ? rows.row(v) : 0) * krow + c * 8, live);
        }
    }
    if (!a.values_in_keys) {
      const int c = tid & ((1 << vlsh) - 1);
      __nv_bfloat16* dst = s_v + (t & 1) * KT * vld + c * 8;
      if (c < vpieces)
        for (int r = tid >> vlsh; r < KT; r += kThreads >> vlsh) {
          const int v = t * KT + r;
          const bool live = v < keys.count;
          cp16z(dst + r * vld, vc + (size_t)(live ? rows.row(v) : 0) * vrow + c * 8, live);
        }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int tiles = (keys.count + KT - 1) / KT;
  const int t0 = (int)((int64_t)tiles * split / sh.splits), t1 = (int)((int64_t)tiles * (split + 1) / sh.splits);
  {
    const int c = tid & ((1 << klsh) - 1);
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q);
    if (c < kpieces)
      for (int i = tid >> klsh; i < M; i += kThreads >> klsh) {
        const bool live = i < np;
        const int p = p0 + (live ? i : 0), qi = p / gq;
        cp16z(s_q + i * ld + c * 8, q + ((size_t)(row0 + qi) * a.heads + kv * gq + p - qi * gq) * a.dpad + c * 8, live);
      }
  }
  if (t0 < t1) fetch(t0);
  else asm volatile("cp.async.commit_group;" ::: "memory");
  // this thread's two rows of the warp's sixteen
  int qpos[2], lo[2], head[2], qrow[2];
  float slope[2];
  bool live[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int i = wr * 16 + (lane >> 2) + 8 * e, p = p0 + i, qi = p / gq;
    live[e] = i < np;
    qrow[e] = row0 + qi;
    head[e] = kv * gq + p - qi * gq;
    qpos[e] = pos_r + qi;
    lo[e] = run_start(a, qpos[e]);
    slope[e] = live[e] && a.slopes ? a.slopes[head[e]] * kLog2E : 0.f;
  }
  const int lo_last = run_start(a, last);
  const float scale2 = a.softcap > 0.f ? 0.f : a.scale * kLog2E;
  const float cap_in = a.softcap > 0.f ? 2.f * kLog2E * a.scale / a.softcap : 0.f, cap_out = a.softcap * kLog2E;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float acc[NV][4];
#pragma unroll
  for (int n = 0; n < NV; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i] = 0.f;
  const int cw = ((a.vpad + WN - 1) / WN + 15) & ~15, col0 = wc * cw, ncol = min(cw, a.vpad - col0);   // the warp's value columns

  for (int t = t0; t < t1; ++t) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                       // tile t is here, nobody reads tile t - 1 or its weights any more
    if (t + 1 < t1) fetch(t + 1);
    const __nv_bfloat16* k = s_k + (t & 1) * KT * ld + wc * KW * ld;
    float s[NS][4];
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) s[j][i] = 0.f;
#pragma unroll 4
    for (int c = 0; c < a.dpad; c += 16) {
      uint32_t qa[4];
      ldm4(qa, s_q + (wr * 16 + (lane & 15)) * ld + c + (lane >> 4) * 8);
      if constexpr (NS == 1) {
        uint32_t kb[2];
        ldm2(kb, k + (lane & 7) * ld + c + ((lane >> 3) & 1) * 8);
        mma16816(s[0], qa, kb[0], kb[1]);
      } else {
#pragma unroll
        for (int j = 0; j < NS; j += 2) {
          uint32_t kb[4];
          ldm4(kb, k + (j * 8 + (lane & 7) + ((lane >> 4) << 3)) * ld + c + ((lane >> 3) & 1) * 8);
          mma16816(s[j], qa, kb[0], kb[1]);
          mma16816(s[j + 1], qa, kb[2], kb[3]);
        }
      }
    }
    // s[j][2 e + i]: row e, key 8 j + 2 (lane & 3) + i of the warp's
    const int v0 = t * KT;
    const bool all_seen = v0 >= keys.nk && v0 + KT <= keys.count && keys.position(v0 + KT - 1) <= first && keys.position(v0) >= lo_last;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int v = v0 + wc * KW + j * 8 + (lane & 3) * 2 + i, p = keys.position(v);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float x = s[j][2 * e + i];
          if (a.softcap > 0.f) x = fmaf(-2.f * cap_out, __fdividef(1.f, exp2f(x * cap_in) + 1.f), cap_out);   // tanh z = 1 - 2 / (e^2z + 1)
          else x *= scale2;
          x = fmaf(-slope[e], (float)(qpos[e] - p), x);
          if (!all_seen && !(v < keys.count && p <= qpos[e] && (p >= lo[e] || p < a.keep_first))) x = -INFINITY;
          s[j][2 * e + i] = x;
          mx[e] = fmaxf(mx[e], x);
        }
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
      if ((lane & 3) == 0) s_max[wc * M + wr * 16 + (lane >> 2) + 8 * e] = mx[e];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float mn = m[e];
#pragma unroll
      for (int w = 0; w < WN; ++w) mn = fmaxf(mn, s_max[w * M + wr * 16 + (lane >> 2) + 8 * e]);
      const float base = mn == -INFINITY ? 0.f : mn;   // nothing seen yet: weights exp(-inf) = 0
      alpha[e] = exp2f(m[e] - base);
      m[e] = mn;
      float sum = 0.f;
      __nv_bfloat16* pr = s_p + (wr * 16 + (lane >> 2) + 8 * e) * PLD + wc * KW + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < NS; ++j) {
        const float w0 = exp2f(s[j][2 * e] - base), w1 = exp2f(s[j][2 * e + 1] - base);
        sum += w0 + w1;
        const __nv_bfloat162 hi = __floats2bfloat162_rn(w0, w1);
        const float2 hf = __bfloat1622float2(hi);
        *reinterpret_cast<__nv_bfloat162*>(pr + j * 8) = hi;
        *reinterpret_cast<__nv_bfloat162*>(pr + M * PLD + j * 8) = __floats2bfloat162_rn(w0 - hf.x, w1 - hf.y);
      }
      l[e] = fmaf(l[e], alpha[e], sum);
    }
    __syncthreads();
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[n][i] *= alpha[i >> 1];
    }
    const __nv_bfloat16* vt = s_v + (t & 1) * KT * vld + col0;
#pragma unroll
    for (int kk = 0; kk < KT; kk += 16) {
      uint32_t hi[4], rest[4];
      const __nv_bfloat16* pp = s_p + (wr * 16 + (lane & 15)) * PLD + kk + (lane >> 4) * 8;
      ldm4(hi, pp);
      ldm4(rest, pp + M * PLD);
#pragma unroll
      for (int n = 0; n < NV; n += 2) {
        if (n * 8 >= ncol) break;
        uint32_t vb[4];   // V is [key][column]: (keys 0-7, cols 0-7) (keys 8-15, cols 0-7) (keys 0-7, cols 8-15) ...
        ldm4t(vb, vt + (kk + (lane & 15)) * vld + n * 8 + (lane >> 4) * 8);
        mma16816(acc[n], hi, vb[0], vb[1]);
        mma16816(acc[n + 1], hi, vb[2], vb[3]);
        mma16816(acc[n], rest, vb[0], vb[1]);
        mma16816(acc[n + 1], rest, vb[2], vb[3]);
      }
    }
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  // the rows' sums over the warps side by side
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    if ((lane & 3) == 0) s_max[wc * M + wr * 16 + (lane >> 2) + 8 * e] = l[e];
  }
  __syncthreads();
  const bool whole = sh.splits == 1;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    if (!live[e]) continue;
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < WN; ++w) sum += s_max[w * M + wr * 16 + (lane >> 2) + 8 * e];
    float f = 1.f;
    if (whole) {
      f = sum > 0.f ? 1.f / sum : 0.f;
      if (a.gate) f *= a.gate[(size_t)qrow[e] * a.heads + head[e]];
    }
    const size_t part = ((size_t)split * a.r.rows + qrow[e]) * a.heads + head[e];
    if (!whole && wc == 0 && (lane & 3) == 0) a.part_ml[part] = make_float2(m[e], sum);
    float* dst = a.parts + part * a.vdim;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      if (n * 8 >= ncol) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int c = col0 + n * 8 + (lane & 3) * 2 + i;
        if (c >= a.vdim) continue;
        if (whole) flash_store_column<true>(a, qrow[e], head[e], c, acc[n][2 * e + i] * f);
        else dst[c] = acc[n][2 * e + i];
      }
    }
    if (whole && wc == 0)
      for (int c = a.vdim + (lane & 3); c < flash_column_limit(a, head[e]); c += 4) flash_store_column<true>(a, qrow[e], head[e], c, 0.f);
  }
}

__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], uint32_t at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}

// The 8 x 8 matrix of 16-bit elements that a warp holds (row lane / 4, columns 2 (lane & 3) and the next), transposed.
__device__ __forceinline__ uint32_t transposed(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}
__device__ __forceinline__ uint32_t pack2(float x, float y) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
  return *reinterpret_cast<const uint32_t*>(&v);
}

constexpr int kDecodeKeys = 32;   // keys a warp takes at a time
constexpr int kDecodeHeads = 8;

// grid (splits, kv heads, rows); DT: at most 16 DT elements of a key, of a value (EXACT: that many of both)
template <int DT, bool EXACT>
__global__ void __launch_bounds__(kThreads) flash_decode_kernel(const FlashArgs a, const FlashShape sh) {
  extern __shared__ __align__(16) unsigned char s_raw[];
  constexpr int KT = kDecodeKeys, NH = kDecodeHeads;
  const int gq = a.heads / a.kv_heads, kv = (int)blockIdx.y, r = (int)blockIdx.z, split = (int)blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = (int)blockDim.x >> 5;
  const int ld = EXACT ? 16 * DT + 8 : a.dpad + 8, vld = EXACT ? 16 * DT + 8 : a.vpad + 8;
  __nv_bfloat16* s_k = reinterpret_cast<__nv_bfloat16*>(s_raw) + (size_t)warp * 2 * KT * (ld + vld);   // the warp's [2][KT][ld], [2][KT][vld]
  __nv_bfloat16* s_v = s_k + 2 * KT * ld;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const BlockKeys keys(pos, pos, a.window, a.keep_first, a.chunk);
  const int krow = a.kv_heads * a.dpad, vrow = a.kv_heads * a.vpad;
  const size_t slot = pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(a.k_cache) + slot * krow + (size_t)kv * a.dpad;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(a.v_cache) + slot * vrow + (size_t)kv * a.vpad;
  const int tiles = (keys.count + KT - 1) / KT;
  const int t0 = (int)((int64_t)tiles * split / sh.splits), t1 = (int)((int64_t)tiles * (split + 1) / sh.splits);
  // 32 rows of `pieces` 16-byte pieces each; row v of a whole tile in one piece of the cache is `row` elements behind row v - 1
  auto rows_in = [&](__nv_bfloat16* dst, int dld, const __nv_bfloat16* src, int row, int pieces, const RunRows& rr, int v0, bool one_piece) {
    int y = lane / pieces, c = lane - y * pieces;
    const int dy = 32 / pieces, dc = 32 - dy * pieces;
    if (EXACT && one_piece) {   // 2 DT pieces: whole rows at a time
      constexpr int P = 2 * DT, DY = 32 / P;
      const __nv_bfloat16* s0 = src + (size_t)rr.row(v0) * row + (size_t)(uint32_t)(lane / P * row) + (lane % P) * 8;
      uint32_t d0 = smem_addr(dst + lane / P * (16 * DT + 8) + (lane % P) * 8);
      const int64_t step = (int64_t)DY * row;
#pragma unroll
      for (int i = 0; i < P; ++i) {
        cp16(d0 + (uint32_t)(i * DY * (16 * DT + 8) * 2), s0);
        s0 += step;
      }
    } else if (one_piece) {
      const __nv_bfloat16* s0 = src + (size_t)rr.row(v0) * row;
      for (int i = 0; i < pieces; ++i) {
        cp16z(dst + y * dld + c * 8, s0 + (size_t)(uint32_t)(y * row) + c * 8, true);
        y += dy;
        c += dc;
        if (c >= pieces) { c -= pieces; ++y; }
      }
    } else {
      for (int i = 0; i < pieces; ++i) {
        const bool live = v0 + y < keys.count;
        cp16z(dst + y * dld + c * 8, src + (size_t)(live ? rr.row(v0 + y) : 0) * row + c * 8, live);
        y += dy;
        c += dc;
        if (c >= pieces) { c -= pieces; ++y; }
      }
    }
  };
  auto fetch = [&](int t, int buf) {
    const int v0 = t * KT;
    const RunRows rr(keys, a.geom, v0);
    const bool one_piece = v0 + KT <= keys.count && rr.row(v0 + KT - 1) - rr.row(v0) == KT - 1;
    rows_in(s_k + buf * KT * ld, ld, kc, krow, a.dpad >> 3, rr, v0, one_piece);
    rows_in(s_v + buf * KT * vld, vld, vc, vrow, a.vpad >> 3, rr, v0, one_piece);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 + warp < t1) fetch(t0 + warp, 0);
  // the queries as the eight columns: element (k, head) with head lane / 4, k 2 (lane & 3) and the next, and 8 on
  uint32_t qb[DT][2];
  {
    const int h = lane >> 2;
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + ((size_t)r * a.heads + kv * gq + (h < gq ? h : 0)) * a.dpad + (lane & 3) * 2;
#pragma unroll
    for (int ks = 0; ks < DT; ++ks) {
      const bool live = h < gq && ks * 16 < a.dpad;
      qb[ks][0] = live ? *reinterpret_cast<const uint32_t*>(q + ks * 16) : 0u;
      qb[ks][1] = live ? *reinterpret_cast<const uint32_t*>(q + ks * 16 + 8) : 0u;
    }
  }
  float slope[2], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};   // of heads 2 (lane & 3) and the next
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    const int h = (lane & 3) * 2 + y;
    slope[y] = a.slopes && h < gq ? a.slopes[kv * gq + h] * kLog2E : 0.f;
  }
  const float scale2 = a.scale * kLog2E, cap_in = a.softcap > 0.f ? 2.f * kLog2E * a.scale / a.softcap : 0.f, cap = a.softcap * kLog2E;
  float acc[DT][4];
#pragma unroll
  for (int n = 0; n < DT; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[n][i] = 0.f;
  int buf = 0;
  for (int t = t0 + warp; t < t1; t += nw, buf ^= 1) {
    if (t + nw < t1) {
      fetch(t + nw, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncwarp();
    const __nv_bfloat16 *k = s_k + buf * KT * ld, *v = s_v + buf * KT * vld;
    float d[2][4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int i = 0; i < 4; ++i) d[x][i] = 0.f;
    const uint32_t k_at = smem_addr(k + (lane & 15) * ld + (lane >> 4) * 8), k_half = (uint32_t)ld * 32;
#pragma unroll
    for (int ks = 0; ks < DT; ++ks) {
      if (!EXACT && ks * 16 >= a.dpad) break;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        uint32_t ka[4];
        ldm4(ka, k_at + (uint32_t)x * k_half + (uint32_t)(ks * 32));
        mma16816(d[x], ka, qb[ks][0], qb[ks][1]);
      }
    }
    // d[x][2 z + y]: key 16 x + lane / 4 + 8 z, head 2 (lane & 3) + y.  Every numbered key of the row's own block is seen.
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        const int n = t * KT + x * 16 + (lane >> 2) + 8 * z;
        const float dist = (float)(pos - keys.position(n));
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          float s = d[x][2 * z + y];
          if (a.softcap > 0.f) s = fmaf(-2.f * cap, __fdividef(1.f, exp2f(s * cap_in) + 1.f), cap);
          else s *= scale2;
          s = n < keys.count ? fmaf(-slope[y], dist, s) : -INFINITY;
          d[x][2 * z + y] = s;
          mx[y] = fmaxf(mx[y], s);
        }
      }
    float alpha[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
#pragma unroll
      for (int o = 16; o > 2; o >>= 1) mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], o));
      const float mn = fmaxf(m[y], mx[y]);   // a tile holds at least one visible key
      alpha[y] = exp2f(m[y] - mn);
      m[y] = mn;
      float sum = 0.f;
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int z = 0; z < 2; ++z) {
          const float w = exp2f(d[x][2 * z + y] - mn);
          d[x][2 * z + y] = w;
          sum += w;
        }
      l[y] = fmaf(l[y], alpha[y], sum);
    }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int n = 0; n < DT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[n][i] *= alpha[i & 1];
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {   // 16 keys: weights in two pieces, [key][head] -> [head][key]
      uint32_t hi[2], rest[2];
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        const float w0 = d[x][2 * z], w1 = d[x][2 * z + 1];
        const uint32_t p = pack2(w0, w1);
        hi[z] = transposed(p);
        rest[z] = transposed(pack2(w0 - __uint_as_float(p << 16), w1 - __uint_as_float(p & 0xFFFF0000u)));
      }
      const uint32_t v_at = smem_addr(v + (x * 16 + (lane & 7) + (lane >> 4) * 8) * vld + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int n = 0; n < DT; ++n) {
        if (!EXACT && n * 16 >= a.vpad) break;
        uint32_t va[4];   // 16 columns x 16 keys out of [key][column]
        ldm4t(va, v_at + (uint32_t)(n * 32));
        mma16816(acc[n], va, hi[0], hi[1]);
        mma16816(acc[n], va, rest[0], rest[1]);
      }
    }
    __syncwarp();
  }
  // ---- the warps' shares ----
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
#pragma unroll
  for (int y = 0; y < 2; ++y)
#pragma unroll
    for (int o = 16; o > 2; o >>= 1) l[y] += __shfl_xor_sync(0xffffffffu, l[y], o);
  float2* s_ml = reinterpret_cast<float2*>(s_raw);                 // [warps][NH]
  float* s_o = reinterpret_cast<float*>(s_ml + nw * NH);           // [warps][NH][vpad + 4]
  const int old = a.vpad + 4;
  if (lane < 4)
#pragma unroll
    for (int y = 0; y < 2; ++y) s_ml[warp * NH + lane * 2 + y] = make_float2(m[y], l[y]);
#pragma unroll
  for (int n = 0; n < DT; ++n) {
    if (n * 16 >= a.vpad) break;
#pragma unroll
    for (int i = 0; i < 4; ++i) {   // column lane / 4 + 8 (i / 2), head 2 (lane & 3) + (i & 1)
      const int h = (lane & 3) * 2 + (i & 1);
      if (h < gq) s_o[(warp * NH + h) * old + n * 16 + (lane >> 2) + (i >> 1) * 8] = acc[n][i];
    }
  }
  __syncthreads();
  const bool whole = sh.splits == 1;
  for (int h = warp; h < gq; h += nw) {
    const int head = kv * gq + h;
    float mm = -INFINITY, sum = 0.f;
    for (int w = 0; w < nw; ++w) mm = fmaxf(mm, s_ml[w * NH + h].x);
    for (int w = 0; w < nw; ++w) {
      const float2 p = s_ml[w * NH + h];
      if (p.x != -INFINITY) sum = fmaf(p.y, exp2f(p.x - mm), sum);
    }
    float f = 1.f;
    if (whole) {
      f = sum > 0.f ? 1.f / sum : 0.f;
      if (a.gate) f *= a.gate[(size_t)r * a.heads + head];
    }
    const size_t part = ((size_t)split * a.r.rows + r) * a.heads + head;
    if (!whole && lane == 0) a.part_ml[part] = make_float2(mm, sum);
    const int limit = whole ? flash_column_limit(a, head) : a.vdim;
    for (int c = lane; c < limit; c += 32) {
      float o = 0.f;
      if (c < a.vdim)
        for (int w = 0; w < nw; ++w) {
          const float x = s_ml[w * NH + h].x;
          if (x != -INFINITY) o = fmaf(s_o[(w * NH + h) * old + c], exp2f(x - mm), o);
        }
      if (whole) flash_store_column<true>(a, r, head, c, o * f);
      else a.parts[part * a.vdim + c] = o;
    }
  }
}

size_t decode_warp_bytes(const FlashArgs& a) { return (size_t)2 * kDecodeKeys * (a.dpad + a.vpad + 16) * 2; }

// Merges the shares of a row's keys.  A lane has four columns, each of W warps every W-th share; what they add up is
// summed over the warps.  grid (heads, rows, columns / 128)
template <int W>
__global__ void __launch_bounds__(W * 32) flash_merge_kernel(const FlashArgs a, const int splits) {
  constexpr int T = W * 32, AHEAD = 8;   // shares whose columns are requested before the weights are known
  __shared__ float s_w[kMaxSplits], s_red[W], s_sum[W];
  __shared__ float4 s_acc[W][32];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = (int)blockIdx.x, r = (int)blockIdx.y, c = (int)blockIdx.z * 128 + lane * 4;
  grid_dep_launch();
  grid_dep_wait();
  const size_t stride = (size_t)a.r.rows * a.heads, at = (size_t)r * a.heads + h;
  const float* p = a.parts + at * a.vdim + c;
  auto load = [&](int z) {
    const float* q = p + (size_t)z * stride * a.vdim;
    if (a.vdim % 4 == 0) return c < a.vdim ? *reinterpret_cast<const float4*>(q) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(c < a.vdim ? q[0] : 0.f, c + 1 < a.vdim ? q[1] : 0.f, c + 2 < a.vdim ? q[2] : 0.f, c + 3 < a.vdim ? q[3] : 0.f);
  };
  float4 v[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
    if (warp + i * W < splits) v[i] = load(warp + i * W);
  float m = -INFINITY;
  for (int z = tid; z < splits; z += T) m = fmaxf(m, a.part_ml[z * stride + at].x);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  if (lane == 0) s_red[warp] = m;
  __syncthreads();
#pragma unroll
  for (int w = 0; w < W; ++w) m = fmaxf(m, s_red[w]);
  float l = 0.f;
  for (int z = tid; z < splits; z += T) {
    const float2 q = a.part_ml[z * stride + at];
    const float w = q.x == -INFINITY ? 0.f : exp2f(q.x - m);   // a share that saw nothing left zeros
    s_w[z] = w;
    l = fmaf(w, q.y, l);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (lane == 0) s_sum[warp] = l;
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  auto add = [&](float w, float4 x) { acc = make_float4(fmaf(w, x.x, acc.x), fmaf(w, x.y, acc.y), fmaf(w, x.z, acc.z), fmaf(w, x.w, acc.w)); };
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
    if (warp + i * W < splits) add(s_w[warp + i * W], v[i]);
  for (int z = warp + AHEAD * W; z < splits; z += W) add(s_w[z], load(z));
  s_acc[warp][lane] = acc;
  __syncthreads();
  if (warp != 0) return;
  l = 0.f;
#pragma unroll
  for (int w = 0; w < W; ++w) l += s_sum[w];
  float f = l > 0.f ? 1.f / l : 0.f;
  if (a.gate) f *= a.gate[at];
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int w = 0; w < W; ++w) add(f, s_acc[w][lane]);
  const float o[4] = {acc.x, acc.y, acc.z, acc.w};
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (c + i < flash_column_limit(a, h)) flash_store_column<true>(a, r, h, c + i, c + i < a.vdim ? o[i] : 0.f);
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
}

// grid (kv heads * groups of four of their query heads, rows)
template <typename T>
__global__ void __launch_bounds__(kThreads) flash_simple_kernel(const FlashArgs a) {
  extern __shared__ __align__(16) float s_f[];
  constexpr int HG = 4, KT = 32;
  __shared__ float s_s[HG][KT], s_alpha[HG], s_l[HG];
  __shared__ int s_row[KT];
  const int gq = a.heads / a.kv_heads, groups = (gq + HG - 1) / HG;
  const int kv = (int)blockIdx.x / groups, h0 = kv * gq + ((int)blockIdx.x - kv * groups) * HG, nh = min(HG, (kv + 1) * gq - h0);
  const int r = (int)blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* s_q = s_f;                    // [HG][dpad]
  float* s_o = s_q + HG * a.dpad;      // [HG][vdim]
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const VisibleRange vr(pos, a.window, a.keep_first, a.chunk);
  const int nv = vr.count();
  const size_t slot = pos < 0 ? 0 : (size_t)a.r.slots[r];
  const int krow = a.kv_heads * a.dpad, vrow = a.values_in_keys ? krow : a.kv_heads * a.vpad;
  const T* kc = static_cast<const T*>(a.k_cache) + slot * a.geom.rows * (size_t)krow + (size_t)kv * a.dpad;
  const T* vc = a.values_in_keys ? kc : static_cast<const T*>(a.v_cache) + slot * a.geom.rows * (size_t)vrow + (size_t)kv * a.vpad;
  const T* q = static_cast<const T*>(a.q) + ((size_t)r * a.heads + h0) * a.dpad;
  for (int i = tid; i < nh * a.dpad; i += kThreads) s_q[i] = (float)q[i];
  for (int i = tid; i < nh * a.vdim; i += kThreads) s_o[i] = 0.f;
  float m = -INFINITY, l = 0.f;        // of head `warp`, in warps 0..nh-1
  for (int t = 0; t < nv; t += KT) {
    const int nj = min(KT, nv - t);
    if (tid < KT) s_row[tid] = a.geom.row_of(vr.position(min(t + tid, nv - 1)));
    __syncthreads();
    {
      const int j = tid >> 3, part = tid & 7;
      const T* k = kc + (size_t)s_row[j] * krow;
      float d[HG] = {0.f, 0.f, 0.f, 0.f};
      for (int c = part * 4; c < a.dpad; c += 32) {
        const float4 x = load4(k + c);
#pragma unroll
        for (int h = 0; h < HG; ++h)
          if (h < nh) {
            const float4 y = load4(s_q + h * a.dpad + c);
            d[h] = fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, d[h]))));
          }
      }
#pragma unroll
      for (int h = 0; h < HG; ++h) {
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) d[h] += __shfl_xor_sync(0xffffffffu, d[h], o);
        if (part == 0 && h < nh) {
          float x = d[h] * a.scale;
          if (a.softcap > 0.f) x = a.softcap * tanhf(x / a.softcap);
          if (a.slopes) x -= a.slopes[h0 + h] * (float)(pos - vr.position(t + j));
          s_s[h][j] = j < nj ? x : -INFINITY;
        }
      }
    }
    __syncthreads();
    if (warp < nh) {
      const float x = s_s[warp][lane];
      float mx = x;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float mn = fmaxf(m, mx), alpha = expf(m - mn), w = expf(x - mn);   // a tile holds at least one visible key
      float sum = w;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      l = fmaf(l, alpha, sum);
      m = mn;
      s_s[warp][lane] = w;
      if (lane == 0) s_alpha[warp] = alpha;
    }
    __syncthreads();
    for (int c = tid; c < a.vdim; c += kThreads) {
      float o[HG];
#pragma unroll
      for (int h = 0; h < HG; ++h) o[h] = h < nh ? s_o[h * a.vdim + c] * s_alpha[h] : 0.f;
      for (int j = 0; j < nj; ++j) {
        const float v = (float)vc[(size_t)s_row[j] * vrow + c];
#pragma unroll
        for (int h = 0; h < HG; ++h) o[h] = h < nh ? fmaf(s_s[h][j], v, o[h]) : 0.f;
      }
#pragma unroll
      for (int h = 0; h < HG; ++h)
        if (h < nh) s_o[h * a.vdim + c] = o[h];
    }
    __syncthreads();
  }
  if (warp < nh && lane == 0) s_l[warp] = l;
  __syncthreads();
  for (int h = 0; h < nh; ++h) {
    float f = s_l[h] > 0.f ? 1.f / s_l[h] : 0.f;
    if (a.gate) f *= a.gate[(size_t)r * a.heads + h0 + h];
    for (int c = tid; c < flash_column_limit(a, h0 + h); c += kThreads)
      flash_store_column<sizeof(T) == 2>(a, r, h0 + h, c, c < a.vdim ? s_o[h * a.vdim + c] * f : 0.f);
  }
}

template <typename T>
tb_status launch_simple(const FlashArgs& a, cudaStream_t st, int* launches) {
  const int gq = a.heads / a.kv_heads;
  const size_t smem = 4 * (size_t)(a.dpad + a.vdim) * sizeof(float);
  if (smem > 200 * 1024) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: attention with heads of size %d/%d", a.dim, a.vdim);
  ++*launches;
  return launch_kernel(flash_simple_kernel<T>, dim3((unsigned)(a.kv_heads * ((gq + 3) / 4)), (unsigned)a.r.rows), dim3(kThreads), smem, st, a.pdl, 1, a);
}

size_t mma_bytes(const FlashArgs& a, int mg, int kt) {
  const size_t m = 16 * (size_t)mg, ld = (size_t)a.dpad + 8, vld = a.values_in_keys ? 0 : (size_t)a.vpad + 8;
  return 2 * (m * ld + 2 * kt * ld + 2 * kt * vld + 2 * m * (kt + 8)) + 4 * (8 / mg) * m;
}
constexpr size_t kSmemMax = 226 * 1024;

using FlashKernel = void (*)(FlashArgs, FlashShape);
// The kernel with at least nv 8-column tiles per warp; null: none.
FlashKernel pick_kernel(int mg, int nv, int kt) {
  if (mg == 1 && kt == 64) return nv <= 2 ? flash_mma_kernel<1, 2, 64> : nv <= 4 ? flash_mma_kernel<1, 4, 64> : nv <= 8 ? flash_mma_kernel<1, 8, 64> : nullptr;
  if (mg == 2 && kt == 64)
    return nv <= 4 ? flash_mma_kernel<2, 4, 64> : nv <= 8 ? flash_mma_kernel<2, 8, 64> : nv <= 16 ? flash_mma_kernel<2, 16, 64> : nullptr;
  if (mg == 2 && kt == 32) return nv <= 8 ? flash_mma_kernel<2, 8, 32> : nv <= 16 ? flash_mma_kernel<2, 16, 32> : nullptr;
  if (mg == 4 && kt == 64)
    return nv <= 4 ? flash_mma_kernel<4, 4, 64> : nv <= 8 ? flash_mma_kernel<4, 8, 64> : nv <= 16 ? flash_mma_kernel<4, 16, 64> : nullptr;
  if (mg == 4 && kt == 32) return nv <= 16 ? flash_mma_kernel<4, 16, 32> : nv <= 32 ? flash_mma_kernel<4, 32, 32> : nullptr;
  return nullptr;
}

}  // namespace

tb_status launch_flash_attention(Precision p, const FlashArgs& a, cudaStream_t st, int* launches) {
  if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dpad % 16 || a.vpad % 16 || (a.values_in_keys && (a.kv_heads != 1 || a.vpad > a.dpad)))
    return fail(TB_ERR_SHAPE, "flash attention: bad shape");
  if (p == Precision::kF32) return launch_simple<float>(a, st, launches);
  const int gq = a.heads / a.kv_heads, rows = a.r.rows;
  auto merge = [&](int splits) -> tb_status {
    ++*launches;
    if (splits == 1) return TB_OK;
    ++*launches;
    const int cols = a.out_per_head ? a.out.kp : a.out.kp - (a.heads - 1) * a.vdim;
    const dim3 grid((unsigned)a.heads, (unsigned)rows, (unsigned)((cols + 127) / 128));
    if (splits <= 8) return launch_kernel(flash_merge_kernel<1>, grid, dim3(32), 0, st, a.pdl, 1, a, splits);
    if (splits <= 32) return launch_kernel(flash_merge_kernel<4>, grid, dim3(128), 0, st, a.pdl, 1, a, splits);
    return launch_kernel(flash_merge_kernel<8>, grid, dim3(256), 0, st, a.pdl, 1, a, splits);
  };
  if (flash_tc5_supported(a)) {
    int splits = 1;
    TB_TRY(launch_flash_tc5(a, st, &splits));
    return merge(splits);
  }
  if (flash_latent_supported(a)) {
    int splits = 1;
    TB_TRY(launch_flash_latent(a, st, &splits));
    return merge(splits);
  }
  if (!a.one_sequence && !a.values_in_keys && gq <= kDecodeHeads && a.dpad <= 256 && a.vpad <= 256) {
    // three CTAs per SM, or one of one warp
    const size_t per = decode_warp_bytes(a);   // also holds a warp's merge: 8 (vpad + 4) floats and its statistics
    int warps = (int)(72 * 1024 / per);
    warps = warps < 1 ? 1 : (warps > 8 ? 8 : warps);
    const int64_t tiles = (a.max_visible + kDecodeKeys - 1) / kDecodeKeys;
    FlashShape sd;
    int64_t splits = 3 * (int64_t)sm_count() / ((int64_t)rows * a.kv_heads);
    if (splits > (tiles + warps - 1) / warps) splits = (tiles + warps - 1) / warps;
    if (splits > kMaxSplits) splits = kMaxSplits;
    if (splits > a.part_slots / ((int64_t)rows * a.heads)) splits = a.part_slots / ((int64_t)rows * a.heads);
    sd.splits = splits < 1 ? 1 : (int)splits;
    const int most = a.dpad > a.vpad ? a.dpad : a.vpad;
    const bool exact = a.dpad == a.vpad && (most == 64 || most == 128 || most == 256);
    FlashKernel dec = most <= 64 ? (exact ? flash_decode_kernel<4, true> : flash_decode_kernel<4, false>)
                      : most <= 128 ? (exact ? flash_decode_kernel<8, true> : flash_decode_kernel<8, false>)
                                    : (exact ? flash_decode_kernel<16, true> : flash_decode_kernel<16, false>);
    TB_TRY(launch_kernel(dec, dim3((unsigned)sd.splits, (unsigned)a.kv_heads, (unsigned)rows), dim3((unsigned)warps * 32), per * warps, st, a.pdl, 1, a, sd));
    return merge(sd.splits);
  }
  if (a.key_rows) return fail(TB_ERR_SHAPE, "flash attention: keys in two pieces of %d and %d columns", a.key_cols, a.dim - a.key_cols);
  FlashShape sh;
  sh.run_rows = a.one_sequence ? rows : 1;
  const int runs = a.one_sequence ? 1 : rows;
  const int64_t pairs = (int64_t)sh.run_rows * gq;
  FlashKernel kern = nullptr;
  int mg = pairs <= 16 ? 1 : (pairs <= 32 ? 2 : 4), kt = 0;
  for (; mg <= 4 && kern == nullptr; mg *= 2) {
    const int wn = 8 / mg, nv = (((a.vpad + wn - 1) / wn + 15) & ~15) / 8;
    const int64_t ctas = (pairs + 16 * mg - 1) / (16 * mg) * a.kv_heads * runs;
    // tiles of 32 keys where they alone fit, or where those of 64 are too few for the SMs
    const bool small = mg > 1 && ctas * ((a.max_visible + 63) / 64) < sm_count();
    for (const int k : {small ? 32 : 64, small ? 64 : 32}) {
      if (kern == nullptr && mma_bytes(a, mg, k) <= kSmemMax) {
        kern = pick_kernel(mg, nv, k);
        kt = k;
      }
    }
    if (kern) break;
  }
  if (kern == nullptr) return launch_simple<__nv_bfloat16>(a, st, launches);
  const int pair_tile = 16 * mg;
  sh.tiles = (int)((pairs + pair_tile - 1) / pair_tile);
  const size_t smem = mma_bytes(a, mg, kt);
  const int64_t ctas = (int64_t)sh.tiles * a.kv_heads * runs, slots = (int64_t)sm_count() * (smem <= 112 * 1024 ? 2 : 1);
  int64_t splits = slots / ctas;
  const int64_t ktiles = (a.max_visible + (a.one_sequence ? pair_tile / gq : 0) + kt - 1) / kt;
  if (splits > ktiles) splits = ktiles;
  if (splits > kMaxSplits) splits = kMaxSplits;
  if (splits > a.part_slots / ((int64_t)rows * a.heads)) splits = a.part_slots / ((int64_t)rows * a.heads);
  if (splits < 1) splits = 1;
  sh.splits = (int)splits;
  TB_TRY(launch_kernel(kern, dim3((unsigned)(sh.tiles * sh.splits), (unsigned)a.kv_heads, (unsigned)runs), dim3(kThreads), smem, st, a.pdl, 1, a, sh));
  return merge(sh.splits);
}

int64_t flash_part_slots(int64_t rows, int64_t heads) {
  // every CTA of a wave leaves at most 64 (row, head) pairs, and a step that fills the wave is not split
  const int64_t wave = 2 * (int64_t)sm_count() * 64, step = 2 * rows * heads;
  return wave > step ? wave : step;
}

}  // namespace tb

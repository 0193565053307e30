// The attention of flash_attention.cu for a portion of one sequence in bf16 on tcgen05.
//
// A CTA takes 128 (query, head) pairs of one key/value head against tiles of 128 keys.  Two softmax warpgroups take
// the tiles in turn, each with its own scores and its own output in tensor memory (128 columns each), its own running
// maximum and sum; what they have is merged at the end like two splits of the keys.  Per tile and warpgroup:
//
//   S = Q K^T                scores into tensor memory (both operands K-major, 128-byte swizzle)
//   softmax                  thread = row: cap, bias, mask, weights back over the scores as two bf16 pieces (the second
//                            one what the rounding of the first left)
//   O += P V                 P from tensor memory, V as it lies in the cache ([key][column]: MN-major)
//
// While one warpgroup is at its softmax the tensor core works for the other.  Keys and values come by TMA, panels of 64
// columns by 128 positions, swizzled on the way; tiles begin at multiples of 128 positions, so that one lies in one
// piece in a ring of a multiple of 128 rows too.  Other rings, and keys in pieces of other than 64 columns, come by
// cp.async from three warps.  One thread issues the MMAs.  The output is rescaled only when the maximum has grown by
// more than 8 powers of two; weights stay exact relative to the sum.  Keys may come in two pieces: columns from one
// matrix, the rest (a rotated part that heads share) from another.
#include <climits>
#include <cstring>

#include "dense.cuh"
#include "flash_attention.cuh"
#include "tc5.cuh"
#include "tma_panel.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

using namespace tc5;

constexpr int kM = 128;               // pairs per CTA
constexpr int kKeys = 128;            // keys per tile
constexpr int kPanel = 16384;         // 128 rows of 128 bytes
constexpr int kThreads = 384;         // two softmax warpgroups, one warp for the MMAs, three for the copies
constexpr int kLoaders = 96;
constexpr size_t kSmemMax = 223 * 1024;   // what 227 KB leave beside the static part
constexpr float kLog2E = 1.44269504f;
constexpr float kGrow = 8.f;

__device__ int g_flash_fault = 0;

__device__ __forceinline__ void cp16z(uint32_t dst, const void* src, bool live) {   // zeros when not live
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void tmem_ld32(uint32_t a, float* v) {   // 32 columns of this thread's lane (no wait)
  uint32_t* r = reinterpret_cast<uint32_t*>(v);
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,"
      "%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
        "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]),
        "=r"(r[31])
      : "r"(a)
      : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t a, const uint32_t* r) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(a), "r"(r[0]), "r"(r[1]),
               "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]),
               "r"(r[14]), "r"(r[15])
               : "memory");
}
__device__ __forceinline__ void tmem_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// D (+)= A (tensor memory) * B (shared memory, MN-major: panels of 64 columns, a key per 128-byte row)
__device__ __forceinline__ void mma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint32_t b_lo, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      ".reg .b64 bd;\n\t"
      "setp.ne.b32 p, %5, 0;\n\t"
      "mov.b64 bd, {%2, %3};\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], bd, %4, p;\n\t"
      "}\n" ::"r"(d_tmem),
      "r"(a_tmem), "r"(b_lo), "r"(kDescHi), "r"(idesc), "r"(acc)
      : "memory");
}

struct FlashMaps {
  CUtensorMap k, rest, v;
};

// Rows of keys or values: key v of the block is row base + v, less `ring` from `end` on.
struct Rows {
  const __nv_bfloat16* p;
  int row, base, end, ring;
  __device__ const __nv_bfloat16* at(int v) const {
    int r = base + v;
    if (r >= end) r -= ring;
    return p + (size_t)r * row;
  }
};
__device__ __forceinline__ Rows cache_rows(const FlashArgs& a, const void* cache, int heads, int width, int kv, int slot, int lo) {
  Rows r;
  r.row = heads * width;
  r.p = static_cast<const __nv_bfloat16*>(cache) + (size_t)slot * a.geom.rows * r.row + (size_t)kv * width;
  r.base = a.geom.row_of(lo);
  r.ring = a.geom.ring;
  r.end = a.geom.ring > 0 ? a.geom.ring : INT_MAX;
  return r;
}

// One loader thread's share of a tile: `pieces` 16-byte pieces per row, from `split` on out of the second source; rows from
// `count` on and pieces from `total` on are zeros.
__device__ __forceinline__ void load_tile(uint32_t dst, const Rows& s0, const Rows& s1, int split, int total, int pieces, int v0, int count, int lt) {
  int r = lt / pieces, c = lt - r * pieces;
  const int dr = kLoaders / pieces, dc = kLoaders - dr * pieces;
  for (; r < kKeys;) {
    const int v = v0 + r;
    const bool live = v < count && c < total;
    const __nv_bfloat16* src = c < split || !live ? s0.at(live ? v : 0) + (live ? c * 8 : 0) : s1.at(v) + (c - split) * 8;
    cp16z(dst + (uint32_t)((c >> 3) * kPanel + r * 128 + (((c & 7) ^ (r & 7)) << 4)), src, live);
    r += dr;
    c += dc;
    if (c >= pieces) {
      c -= pieces;
      ++r;
    }
  }
}

// tanh x for |x| <= 1/2: its series, up to x^13 (the next term is below 5e-8).
__device__ __forceinline__ float tanh_series(float x) {
  const float y = x * x;
  float p = fmaf(y, (float)(21844.0 / 6081075.0), (float)(-1382.0 / 155925.0));
  p = fmaf(y, p, (float)(62.0 / 2835.0));
  p = fmaf(y, p, (float)(-17.0 / 315.0));
  p = fmaf(y, p, (float)(2.0 / 15.0));
  p = fmaf(y, p, (float)(-1.0 / 3.0));
  return fmaf(x * y, p, x);
}

// CAP: 0 none, 1 small arguments (|scale q.k / softcap| <= 1/2 by the caller's promise), 2 any.
// grid (tiles * splits, kv heads)
template <int CAP, bool TMA>
__global__ void __launch_bounds__(kThreads, 1) flash_tc5_kernel(const FlashArgs a, const FlashShape sh, const __grid_constant__ FlashMaps maps) {
  extern __shared__ __align__(1024) unsigned char s_raw[];
  __shared__ __align__(8) uint64_t k_full[2], v_full[2], s_ready[2], p_ready[2], pv_done[2], q_full, finished;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  __shared__ float2 s_ml[2][kM];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(s_raw) + 1023) & ~(uintptr_t)1023);
  const int kpieces = a.dpad >> 3, vpieces = a.vpad >> 3, kbytes = (kpieces + 7) / 8 * kPanel, vbytes = (vpieces + 7) / 8 * kPanel;
  const uint32_t q_at = smem_u32(smem), k_at = q_at + kbytes, v_at = k_at + 2 * kbytes;   // [2] tiles each
  const int gq = a.heads / a.kv_heads, kv = (int)blockIdx.y;
  const int split = (int)blockIdx.x % sh.splits, tile = sh.tiles - 1 - (int)blockIdx.x / sh.splits;   // the longest tiles first
  const int p0 = tile * kM, np = min(kM, sh.run_rows * gq - p0);

  if (tid == 0) {
    s_abort = 0;
    for (int w = 0; w < 2; ++w) {
      mbar_init(&k_full[w], TMA ? 1 : kLoaders);
      mbar_init(&v_full[w], TMA ? 1 : kLoaders);
      mbar_init(&s_ready[w], 1);
      mbar_init(&p_ready[w], 128);
      mbar_init(&pv_done[w], 1);
    }
    mbar_init(&q_full, kLoaders);
    mbar_init(&finished, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 8) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  grid_dep_launch();   // after the allocation: kernels behind this one may hold tensor memory while they wait for it
  const uint32_t tmem = s_tmem;
  grid_dep_wait();
  const int pos_r = a.r.pos[0];
  const int first = pos_r + p0 / gq;
  int last = pos_r + (p0 + np - 1) / gq;
  if (a.geom.ring == 0) last = min(last, (int)a.geom.rows - 1);
  const int begin = TMA ? VisibleRange(first, a.window, 0, a.chunk).lo / kKeys * kKeys : VisibleRange(first, a.window, 0, a.chunk).lo;
  const int count = pos_r < 0 ? 0 : last - begin + 1;       // keys from position `begin` on
  const int tiles = (count + kKeys - 1) / kKeys;
  const int t0 = (int)((int64_t)tiles * split / sh.splits), t1 = (int)((int64_t)tiles * (split + 1) / sh.splits);
  const int nj[2] = {(t1 - t0 + 1) / 2, (t1 - t0) / 2};   // tiles t0 + 2 j + w of warpgroup w

  if (warp >= 9) {   // ---- copies ----
    const int lt = tid - 288;
    const int slot = pos_r < 0 ? 0 : a.r.slots[0];
    {   // the queries
      const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q);
      int r = lt / kpieces, c = lt - r * kpieces;
      const int dr = kLoaders / kpieces, dc = kLoaders - dr * kpieces;
      for (; r < kM;) {
        const bool live = r < np;
        const int p = p0 + (live ? r : 0), qi = p / gq;
        cp16z(q_at + (uint32_t)((c >> 3) * kPanel + r * 128 + (((c & 7) ^ (r & 7)) << 4)),
              q + ((size_t)qi * a.heads + kv * gq + p - qi * gq) * a.dpad + c * 8, live);
        r += dr;
        c += dc;
        if (c >= kpieces) {
          c -= kpieces;
          ++r;
        }
      }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    mbar_arrive(&q_full);
    if constexpr (TMA) {
      if (lt == 0) {
        const int kpanels = kbytes / kPanel, vpanels = vbytes / kPanel, kfirst = a.key_rows ? a.key_cols >> 6 : kpanels;
        const size_t slot_row = (size_t)slot * a.geom.rows;
        int k_issued[2] = {0, 0}, v_issued[2] = {0, 0};
        bool ok = true;
        for (int j = 0; ok && j < nj[0]; ++j) {
          for (int w = 0; w < 2; ++w) {
            if (j >= nj[w]) continue;
            if (j > 0 && !(ok = mbar_wait(&s_ready[w], (uint32_t)(j - 1) & 1u, &s_abort, &g_flash_fault))) break;
            const int k0 = begin + (t0 + 2 * j + w) * kKeys, crow = (int)(slot_row + a.geom.row_of(k0));
            k_issued[w] = j + 1;
            mbar_expect_tx(&k_full[w], (uint32_t)kbytes);
            for (int c = 0; c < kpanels; ++c) {
              const uint32_t dst = k_at + (uint32_t)(w * kbytes + c * kPanel);
              if (c >= kfirst) tma_panel(dst, &maps.rest, a.rest_col + (c - kfirst) * 64, crow, smem_u32(&k_full[w]));
              else if (a.key_rows) tma_panel(dst, &maps.k, kv * a.key_cols + c * 64, k0 - a.key_base, smem_u32(&k_full[w]));
              else tma_panel(dst, &maps.k, kv * a.dpad + c * 64, crow, smem_u32(&k_full[w]));
            }
          }
          for (int w = 0; ok && w < 2; ++w) {
            if (j >= nj[w]) continue;
            if (j > 0 && !(ok = mbar_wait(&pv_done[w], (uint32_t)(j - 1) & 1u, &s_abort, &g_flash_fault))) break;
            const int k0 = begin + (t0 + 2 * j + w) * kKeys, crow = (int)(slot_row + a.geom.row_of(k0));
            v_issued[w] = j + 1;
            mbar_expect_tx(&v_full[w], (uint32_t)vbytes);
            for (int c = 0; c < vpanels; ++c)
              tma_panel(v_at + (uint32_t)(w * vbytes + c * kPanel), &maps.v, kv * (a.key_rows ? a.vdim : a.vpad) + c * 64, a.key_rows ? k0 - a.key_base : crow, smem_u32(&v_full[w]));
          }
        }
        if (!ok) {   // copies in flight land before the shared memory is given back: the last one issued per slot
          int no_abort = 0;
          for (int w = 0; w < 2; ++w) {
            if (k_issued[w] > 0) mbar_wait(&k_full[w], (uint32_t)(k_issued[w] - 1) & 1u, &no_abort, &g_flash_fault);
            if (v_issued[w] > 0) mbar_wait(&v_full[w], (uint32_t)(v_issued[w] - 1) & 1u, &no_abort, &g_flash_fault);
          }
        }
      }
    } else {
      Rows ks, ks2, vs;
      const int split_piece = a.key_rows ? a.key_cols >> 3 : kpieces, total = a.dim >> 3;
      if (a.key_rows) {   // written out by position, the rest of a key in the cache
        ks = Rows{static_cast<const __nv_bfloat16*>(a.key_rows) + (size_t)kv * a.key_cols, a.row_stride, begin - a.key_base, INT_MAX, 0};
        vs = Rows{static_cast<const __nv_bfloat16*>(a.value_rows) + (size_t)kv * a.vdim, a.row_stride, begin - a.key_base, INT_MAX, 0};
        ks2 = cache_rows(a, static_cast<const __nv_bfloat16*>(a.k_cache) + a.rest_col, 1, a.cache_row, 0, slot, begin);
      } else {
        ks = ks2 = cache_rows(a, a.k_cache, a.kv_heads, a.dpad, kv, slot, begin);
        vs = cache_rows(a, a.v_cache, a.kv_heads, a.vpad, kv, slot, begin);
      }
      uint64_t* pending = nullptr;   // the load in flight in front of the one being issued
      auto flush = [&] {
        if (!pending) return;
        asm volatile("cp.async.wait_all;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        mbar_arrive(pending);
        pending = nullptr;
      };
      auto freed = [&](uint64_t* bar, int j) {   // the slot's last reader, tile j, is done
        if (mbar_ready(bar, (uint32_t)j & 1u)) return true;
        flush();
        return mbar_wait(bar, (uint32_t)j & 1u, &s_abort, &g_flash_fault);
      };
      auto issued = [&](uint64_t* bar) {
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (pending) {
          asm volatile("cp.async.wait_group 1;" ::: "memory");
          asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
          mbar_arrive(pending);
        }
        pending = bar;
      };
      bool ok = true;
      for (int j = 0; ok && j < nj[0]; ++j) {
        for (int w = 0; ok && w < 2; ++w) {
          if (j >= nj[w]) continue;
          if (j > 0 && !(ok = freed(&s_ready[w], j - 1))) break;
          load_tile(k_at + (uint32_t)(w * kbytes), ks, ks2, split_piece, a.key_rows ? total : kpieces, kpieces, (t0 + 2 * j + w) * kKeys, count, lt);
          issued(&k_full[w]);
        }
        for (int w = 0; ok && w < 2; ++w) {
          if (j >= nj[w]) continue;
          if (j > 0 && !(ok = freed(&pv_done[w], j - 1))) break;
          load_tile(v_at + (uint32_t)(w * vbytes), vs, vs, vpieces, a.key_rows ? a.vdim >> 3 : vpieces, vpieces, (t0 + 2 * j + w) * kKeys, count, lt);
          issued(&v_full[w]);
        }
      }
      flush();
      asm volatile("cp.async.wait_all;" ::: "memory");
    }
  } else if (warp == 8) {
    if (lane == 0) {   // ---- MMA issue ----
      constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kKeys >> 3) << 17) | ((uint32_t)(kM >> 4) << 24);
      const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(a.vpad >> 3) << 17) | ((uint32_t)(kM >> 4) << 24);
      const int ksteps = a.dpad >> 4;
      bool ok = mbar_wait(&q_full, 0u, &s_abort, &g_flash_fault);
      for (int j = 0; ok && j <= nj[0]; ++j)
        for (int w = 0; ok && w < 2; ++w) {
          if (j >= 1 && j - 1 < nj[w]) {   // the output of the tile before
            const uint32_t par = (uint32_t)(j - 1) & 1u;
            ok = mbar_wait(&v_full[w], par, &s_abort, &g_flash_fault) && mbar_wait(&p_ready[w], par, &s_abort, &g_flash_fault);
            if (!ok) break;
            tc_fence_after();
            const uint32_t v_lo = ((v_at + (uint32_t)(w * vbytes)) >> 4) | ((uint32_t)(kPanel >> 4) << 16);
            const uint32_t pt = tmem + (uint32_t)(w * 128), ot = tmem + 256u + (uint32_t)(w * 128);
#pragma unroll
            for (int kk = 0; kk < kKeys / 16; ++kk) {
              const uint32_t at = pt + (uint32_t)((kk >> 1) * 32 + (kk & 1) * 8);   // per 32 keys: 16 columns of the one piece, 16 of the other
              mma_bf16_ts(ot, at, v_lo + (uint32_t)(kk * 128), idesc_o, (j > 1 || kk > 0) ? 1u : 0u);
              mma_bf16_ts(ot, at + 16u, v_lo + (uint32_t)(kk * 128), idesc_o, 1u);
            }
            mma_commit(&pv_done[w]);
          }
          if (j < nj[w]) {
            ok = mbar_wait(&k_full[w], (uint32_t)j & 1u, &s_abort, &g_flash_fault);
            if (!ok) break;
            tc_fence_after();
            const uint32_t q_lo = (q_at >> 4) | (1u << 16), k_lo = ((k_at + (uint32_t)(w * kbytes)) >> 4) | (1u << 16);
            for (int ks = 0; ks < ksteps; ++ks) {
              const uint32_t off = (uint32_t)((ks >> 2) * (kPanel >> 4) + (ks & 3) * 2);
              mma_bf16_ss(tmem + (uint32_t)(w * 128), q_lo + off, k_lo + off, idesc_s, ks > 0 ? 1u : 0u);
            }
            mma_commit(&s_ready[w]);
          }
        }
      mma_commit(&finished);
      int no_abort = 0;
      mbar_wait(&finished, 0u, &no_abort, &g_flash_fault);
    }
  } else {   // ---- softmax: thread = row ----
    const int w = warp >> 2, i = tid & 127, p = p0 + i, qi = p / gq, pos = pos_r + qi;
    const bool row_live = i < np;
    const uint32_t lane_at = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t st = tmem + lane_at + (uint32_t)(w * 128), ot = tmem + lane_at + 256u + (uint32_t)(w * 128);
    const int lo = VisibleRange(pos, a.window, 0, a.chunk).lo, lo_last = VisibleRange(last, a.window, 0, a.chunk).lo;
    const float slope = row_live && a.slopes ? a.slopes[kv * gq + p - qi * gq] * kLog2E : 0.f;
    const float in = CAP == 0 ? a.scale * kLog2E : (CAP == 1 ? a.scale / a.softcap : 2.f * kLog2E * a.scale / a.softcap);
    const float cap = a.softcap * kLog2E;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nj[w]; ++j) {
      ok = mbar_wait(&s_ready[w], (uint32_t)j & 1u, &s_abort, &g_flash_fault);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const int v0 = (t0 + 2 * j + w) * kKeys, k0 = begin + v0;   // position of the tile's first key
      const bool edge = !(k0 + kKeys - 1 <= first && k0 >= lo_last);   // not every row sees every key
      const int jlo = lo - k0, jhi = row_live ? pos - k0 : -1;
      float mx = -INFINITY;
      // 32 columns at a time: few registers, and code that the instruction cache holds
#pragma unroll 1
      for (int q = 0; q < kKeys; q += 32) {
        float s[32];
        tmem_ld32(st + (uint32_t)q, s);
        tmem_wait_ld();
        const float base = -slope * (float)(pos - k0 - q);
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          float x = s[c] * in;
          if (CAP == 1) x = fmaf(cap, tanh_series(x), base);
          else if (CAP == 2) x = fmaf(-2.f * cap, __fdividef(1.f, ex2(x) + 1.f), cap + base);
          else x += base;
          s[c] = fmaf(slope, (float)c, x);
        }
        if (edge) {
#pragma unroll
          for (int c = 0; c < 32; ++c)
            if (q + c < jlo || q + c > jhi) s[c] = -INFINITY;
        }
#pragma unroll
        for (int c = 0; c < 32; ++c) mx = fmaxf(mx, s[c]);
        tmem_st16(st + (uint32_t)q, reinterpret_cast<const uint32_t*>(s));
        tmem_st16(st + (uint32_t)q + 16u, reinterpret_cast<const uint32_t*>(s) + 16);
      }
      tmem_wait_st();
      // the reference the weights are taken against moves only when it must
      const bool grow = mx > m + kGrow || m == -INFINITY;
      const float m1 = grow ? fmaxf(m, mx) : m;
      const float alpha = m == -INFINITY ? 0.f : ex2(m - m1);
      if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f && m != -INFINITY)) {
#pragma unroll 1
        for (int c = 0; c < a.vpad; c += 16) {
          uint32_t r[2][8];
          tmem_ld8(ot + (uint32_t)c, r[0]);
          tmem_ld8(ot + (uint32_t)c + 8, r[1]);
          tmem_wait_ld();
          uint32_t o[16];
#pragma unroll
          for (int x = 0; x < 16; ++x) o[x] = __float_as_uint(__uint_as_float(r[x >> 3][x & 7]) * (m == -INFINITY ? 1.f : alpha));
          tmem_st16(ot + (uint32_t)c, o);
        }
      }
      l *= alpha;
      m = m1;
      const float ref = m == -INFINITY ? 0.f : m;   // nothing seen yet: weights 2^-inf = 0
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll 1
      for (int q = 0; q < kKeys; q += 32) {   // the two pieces of 32 weights take the place of their scores
        float s[32];
        uint32_t hi[16], rest[16];
        tmem_ld32(st + (uint32_t)q, s);
        tmem_wait_ld();
#pragma unroll
        for (int x = 0; x < 16; ++x) {
          const float w0 = ex2(s[2 * x] - ref), w1 = ex2(s[2 * x + 1] - ref);
          sum0 += w0;
          sum1 += w1;
          const __nv_bfloat162 h2 = __floats2bfloat162_rn(w0, w1);
          hi[x] = *reinterpret_cast<const uint32_t*>(&h2);
          const __nv_bfloat162 r2 = __floats2bfloat162_rn(w0 - __uint_as_float(hi[x] << 16), w1 - __uint_as_float(hi[x] & 0xFFFF0000u));
          rest[x] = *reinterpret_cast<const uint32_t*>(&r2);
        }
        tmem_st16(st + (uint32_t)q, hi);
        tmem_st16(st + (uint32_t)q + 16u, rest);
      }
      l += sum0 + sum1;
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(&p_ready[w]);
    }
    if (ok && nj[w] > 0) mbar_wait(&pv_done[w], (uint32_t)(nj[w] - 1) & 1u, &s_abort, &g_flash_fault);
    s_ml[w][i] = make_float2(m, l);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // ---- the two warpgroups' shares, and out ----
  float* s_o = reinterpret_cast<float*>(smem);   // [kM][vpad + 1]
  const int old = a.vpad + 1;
  if (warp < 8) {
    const int w = warp >> 2, i = tid & 127, p = p0 + i, qi = p / gq, head = kv * gq + p - qi * gq;
    const bool row_live = i < np;
    const uint32_t ot = tmem + ((uint32_t)((warp & 3) * 32) << 16) + 256u + (uint32_t)(w * 128);
    const float2 m0 = s_ml[0][i], m1 = s_ml[1][i];
    const float m = fmaxf(m0.x, m1.x);
    float f = s_ml[w][i].x == -INFINITY ? 0.f : ex2(s_ml[w][i].x - m);   // one that saw nothing has left nothing or zeros
    const float l = (m0.x == -INFINITY ? 0.f : m0.y * ex2(m0.x - m)) + (m1.x == -INFINITY ? 0.f : m1.y * ex2(m1.x - m));
    const bool whole = sh.splits == 1;
    if (whole) {
      f *= l > 0.f ? 1.f / l : 0.f;
      if (a.gate && row_live) f *= a.gate[(size_t)qi * a.heads + head];
    }
    const size_t part = ((size_t)split * a.r.rows + qi) * a.heads + head;
    auto columns = [&](auto&& use) {   // eight columns at a time, scaled
      for (int c = 0; c < a.vpad; c += 16) {
        uint32_t r[2][8];
        __syncwarp();
        if (nj[w] > 0) {
          tmem_ld8(ot + (uint32_t)c, r[0]);
          tmem_ld8(ot + (uint32_t)c + 8, r[1]);
          tmem_wait_ld();
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          float v[8];
#pragma unroll
          for (int x = 0; x < 8; ++x) v[x] = f != 0.f && nj[w] > 0 ? __uint_as_float(r[h][x]) * f : 0.f;
          use(c + 8 * h, v);
        }
      }
    };
    if (w == 1 && nj[1] > 0)
      columns([&](int c, const float(&v)[8]) {
#pragma unroll
        for (int x = 0; x < 8; ++x) s_o[i * old + c + x] = v[x];
      });
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (w == 0) {
      columns([&](int c, float(&v)[8]) {
        if (!row_live || c >= a.vdim) return;
        if (nj[1] > 0)
#pragma unroll
          for (int x = 0; x < 8; ++x) v[x] += s_o[i * old + c + x];
        if (!whole) {
          float* dst = a.parts + part * a.vdim + c;
          *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
          return;
        }
        uint32_t u[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * x], v[2 * x + 1]);
          u[x] = *reinterpret_cast<const uint32_t*>(&b);
        }
        *reinterpret_cast<uint4*>(static_cast<unsigned char*>(a.out.data) + image_offset(a.out.mp, qi, head * a.vdim + c)) = make_uint4(u[0], u[1], u[2], u[3]);
      });
      if (row_live && whole)
        for (int c = a.vdim; c < flash_column_limit(a, head); ++c) act_store1<true>(a.out, qi, head * a.vdim + c, 0.f);
      if (row_live && !whole) a.part_ml[part] = make_float2(m, l);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
  }
}

size_t tc5_bytes(int dpad, int vpad) {
  const size_t k = (size_t)(dpad + 63) / 64 * kPanel, v = (size_t)(vpad + 63) / 64 * kPanel, out = (size_t)kM * (vpad + 1) * 4;
  const size_t tiles = 3 * k + 2 * v;
  return (tiles > out ? tiles : out) + 1024;
}

}  // namespace

int flash_fault_flag() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_flash_fault, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

bool flash_tc5_fits(int dpad, int vdim) {
  const int vpad = (int)pad_to(vdim, 16);
  return vdim % 8 == 0 && vpad <= 128 && dpad <= 768 && tc5_bytes(dpad, vpad) <= kSmemMax;
}

bool flash_tc5_supported(const FlashArgs& a) {
  return a.one_sequence && !a.values_in_keys && !a.out_per_head && a.keep_first == 0 && flash_tc5_fits(a.dpad, a.vdim) &&
         (int64_t)a.r.rows * (a.heads / a.kv_heads) >= kM / 2 && (a.key_rows == nullptr || (a.dim % 8 == 0 && a.key_cols % 8 == 0 && a.rest_col % 8 == 0));
}

tb_status launch_flash_tc5(const FlashArgs& a, cudaStream_t st, int* splits_out) {
  const int gq = a.heads / a.kv_heads;
  FlashShape sh;
  sh.run_rows = a.r.rows;
  sh.tiles = (a.r.rows * gq + kM - 1) / kM;
  const int64_t ctas = (int64_t)sh.tiles * a.kv_heads, ktiles = (a.max_visible + kM / gq + kKeys - 1) / kKeys;
  int64_t splits = sm_count() / ctas;
  if (splits > ktiles / 4) splits = ktiles / 4;   // four tiles at least
  if (splits > a.part_slots / ((int64_t)a.r.rows * a.heads)) splits = a.part_slots / ((int64_t)a.r.rows * a.heads);
  if (splits < 1) splits = 1;
  sh.splits = (int)splits;
  *splits_out = sh.splits;
  const dim3 grid((unsigned)(sh.tiles * sh.splits), (unsigned)a.kv_heads);
  const size_t smem = tc5_bytes(a.dpad, a.vpad);
  // unit-norm queries and keys, rounded to bf16: |q . k| <= 1.01 dim
  const int cap = a.softcap <= 0.f ? 0 : (a.unit_norm && 1.01f * fabsf(a.scale) * (float)a.dim <= 0.5f * a.softcap ? 1 : 2);
  FlashMaps maps;
  memset(&maps, 0, sizeof(maps));
  bool tma = a.geom.ring % kKeys == 0 && a.geom.keep == 0 && a.cache_slots > 0;
  if (a.key_rows) {
    const int64_t n = a.key_count;
    tma = tma && a.key_cols % 64 == 0 && a.key_base % kKeys == 0 && tma_panel_map(&maps.k, a.key_rows, (int64_t)a.kv_heads * a.key_cols, n, a.row_stride, kKeys) &&
          tma_panel_map(&maps.v, a.value_rows, (int64_t)a.kv_heads * a.vdim, n, a.row_stride, kKeys) &&
          tma_panel_map(&maps.rest, a.k_cache, a.cache_row, a.cache_slots * a.geom.rows, a.cache_row, kKeys);
  } else {
    const int64_t n = (int64_t)a.cache_slots * a.geom.rows, kw = (int64_t)a.kv_heads * a.dpad, vw = (int64_t)a.kv_heads * a.vpad;
    tma = tma && tma_panel_map(&maps.k, a.k_cache, kw, n, kw, kKeys) && tma_panel_map(&maps.v, a.v_cache, vw, n, vw, kKeys);
  }
  using Kernel = void (*)(FlashArgs, FlashShape, FlashMaps);
  static const Kernel kernels[3][2] = {{flash_tc5_kernel<0, false>, flash_tc5_kernel<0, true>},
                                       {flash_tc5_kernel<1, false>, flash_tc5_kernel<1, true>},
                                       {flash_tc5_kernel<2, false>, flash_tc5_kernel<2, true>}};
  return launch_kernel(kernels[cap][tma ? 1 : 0], grid, dim3(kThreads), smem, st, a.pdl, 1, a, sh, maps);
}

}  // namespace tb

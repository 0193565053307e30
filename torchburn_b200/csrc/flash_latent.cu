// Decode steps of attention over latents (flash_attention.cu: one key/value head shared by all query heads, whose values
// are the first elements of its keys) in bf16 on tcgen05.
//
// A few dozen heads against one row of keys would leave most of a 128-row MMA empty, so keys and value columns are the
// MMA's rows and the heads its columns:
//
//   S^T [64 keys, heads]       = K Q^T      K as it lies in the cache, K-major
//   O^T [value columns, heads] += V^T P^T   the same tile read MN-major: V is K's first columns; P^T from shared memory
//
// 64 keys per tile, tiles by TMA, swizzled, two to four of them in flight.  Four warps hold the scores of 16 keys each (the way
// an MMA of 64 rows leaves them).  Weights are two bf16 pieces, the second one what the rounding of the first left; the
// pieces of the heads are the columns of one MMA, and their outputs are added at the end.  The output is rescaled only
// when a maximum has grown by more than 8 powers of two.  One thread issues the MMAs, scores or outputs, whatever is
// ready.  CTAs that share a row's keys leave parts for the merge.
#include <climits>

#include "flash_attention.cuh"
#include "tc5.cuh"
#include "tma_panel.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

using namespace tc5;

constexpr int kKeys = 64;            // keys per tile
constexpr int kPanel = kKeys * 128;  // 64 columns of a tile
constexpr int kThreads = 192;        // four softmax / output warps, one for TMA, one for the MMAs
constexpr int kStagesMax = 4;
constexpr int kColumns = 512;        // of tensor memory
constexpr float kLog2E = 1.44269504f;
constexpr float kGrow = 8.f;

__device__ int g_latent_fault = 0;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
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
// 16 lanes x 8 columns over the warp: lane / 4 (v0, v1) and 8 lanes on (v2, v3), columns 2 (lane & 3) and the next (no wait)
__device__ __forceinline__ void tmem_ld_tile(uint32_t at, float (&v)[4]) {
  uint32_t r[4];
  asm volatile("tcgen05.ld.sync.aligned.16x256b.x1.b32 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
#pragma unroll
  for (int x = 0; x < 4; ++x) v[x] = __uint_as_float(r[x]);
}
// NH columns of this thread's lane
template <int NH>
__device__ __forceinline__ void tmem_load(uint32_t at, float (&v)[NH]) {
#pragma unroll
  for (int c = 0; c < NH; c += 8) {
    uint32_t r[8];
    tmem_ld8(at + (uint32_t)c, r);
#pragma unroll
    for (int x = 0; x < 8; ++x) v[c + x] = __uint_as_float(r[x]);
  }
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_st8(uint32_t at, const float* v) {
  const uint32_t* r = reinterpret_cast<const uint32_t*>(v);
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(at), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]),
               "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}

struct LatentShape {
  int splits, stages, panels, mtiles, stage_bytes;
};

// grid (splits, groups of NH heads, rows)
template <int NH>
__global__ void __launch_bounds__(kThreads, 1) flash_latent_kernel(const FlashArgs a, const LatentShape sh, const __grid_constant__ CUtensorMap map) {
  extern __shared__ __align__(1024) unsigned char s_raw[];
  __shared__ __align__(8) uint64_t full[kStagesMax], empty[kStagesMax], s_ready[2], p_ready[2], pv_done[2], q_full, finished;
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort, s_grown, s_bad;
  __shared__ __align__(16) float s_max[4][NH], s_ref[NH], s_alpha[NH], s_l[4][NH];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(s_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t k_at = smem_u32(smem), q_at = k_at + (uint32_t)(sh.stages * sh.stage_bytes), p_at = q_at + (uint32_t)(sh.panels * NH * 128);
  const int r = (int)blockIdx.z, h0 = (int)blockIdx.y * NH, nh = min(NH, a.heads - h0), split = (int)blockIdx.x;
  if (tid == 0) {
    s_abort = s_bad = 0;
    for (int s = 0; s < kStagesMax; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int w = 0; w < 2; ++w) {
      mbar_init(&s_ready[w], 1);
      mbar_init(&p_ready[w], 128);
      mbar_init(&pv_done[w], 1);
    }
    mbar_init(&q_full, 128);
    mbar_init(&finished, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  grid_dep_launch();   // after the allocation: kernels behind this one may hold tensor memory while they wait for it
  const uint32_t tmem = s_tmem, o_at = tmem + 2 * NH;
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const int lo = VisibleRange(pos, a.window, 0, a.chunk).lo, begin = lo / kKeys * kKeys;
  const int tiles = pos < 0 ? 0 : (pos - begin) / kKeys + 1;
  const int t0 = (int)((int64_t)tiles * split / sh.splits), n = (int)((int64_t)tiles * (split + 1) / sh.splits) - t0;

  if (warp == 4) {
    if (lane == 0) {   // ---- tiles ----
      const int slot_row = pos < 0 ? 0 : (int)((int64_t)a.r.slots[r] * a.geom.rows);
      int issued = 0;
      for (int i = 0; i < n; ++i) {
        const int s = i % sh.stages;
        if (i >= sh.stages && !mbar_wait(&empty[s], (uint32_t)(i / sh.stages - 1) & 1u, &s_abort, &g_latent_fault)) break;
        mbar_expect_tx(&full[s], (uint32_t)(sh.panels * kPanel));
        const int row = slot_row + a.geom.row_of(begin + (t0 + i) * kKeys);
        for (int c = 0; c < sh.panels; ++c) tma_panel(k_at + (uint32_t)(s * sh.stage_bytes + c * kPanel), &map, c * 64, row, smem_u32(&full[s]));
        issued = i + 1;
      }
      if (issued < n)   // given up: copies in flight land before the shared memory is given back
        for (int i = issued > sh.stages ? issued - sh.stages : 0; i < issued; ++i) {
          int no_abort = 0;
          mbar_wait(&full[i % sh.stages], (uint32_t)(i / sh.stages) & 1u, &no_abort, &g_latent_fault);
        }
    }
  } else if (warp == 5) {
    if (lane == 0) {   // ---- MMA issue ----
      // scores: 64 rows, row k in lane k % 16 + 32 (k / 16); output: 128 rows, MN-major
      constexpr uint32_t shape = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NH >> 3) << 17);
      constexpr uint32_t idesc_s = shape | (4u << 24), idesc_o = (shape + ((uint32_t)(NH >> 3) << 17)) | (1u << 15) | (8u << 24);   // both pieces
      const int ksteps = a.dpad >> 4;
      bool ok = mbar_wait(&q_full, 0u, &s_abort, &g_latent_fault);
      int scored = 0, summed = 0;
      long long idle = 0;
      while (ok && summed < n) {   // whatever is ready first: the output of a tile, or the scores of one up to two ahead
        bool did = false;
        if (summed < scored && mbar_ready(&p_ready[summed & 1], (uint32_t)(summed >> 1) & 1u)) {
          const int t = summed++, s = t % sh.stages;
          tc_fence_after();
          const uint32_t v_lo = ((k_at + (uint32_t)(s * sh.stage_bytes)) >> 4) | ((uint32_t)(kPanel >> 4) << 16);
          const uint32_t p_lo = ((p_at + (uint32_t)((t & 1) * 2 * NH * 128)) >> 4) | (1u << 16);
          for (int mt = 0; mt < sh.mtiles; ++mt)
#pragma unroll
            for (int kk = 0; kk < kKeys / 16; ++kk)
              mma_bf16_ss(o_at + (uint32_t)(mt * 2 * NH), v_lo + (uint32_t)(mt * 2 * (kPanel >> 4) + kk * 128), p_lo + (uint32_t)(kk * 2), idesc_o,
                          (t > 0 || kk > 0) ? 1u : 0u);
          mma_commit(&empty[s]);
          mma_commit(&pv_done[t & 1]);
          did = true;
        }
        if (scored < n && scored < summed + 2 && mbar_ready(&full[scored % sh.stages], (uint32_t)(scored / sh.stages) & 1u)) {
          const int i = scored++, s = i % sh.stages;
          tc_fence_after();
          const uint32_t k_lo = ((k_at + (uint32_t)(s * sh.stage_bytes)) >> 4) | (1u << 16), q_lo = (q_at >> 4) | (1u << 16);
#pragma unroll 4
          for (int ks = 0; ks < ksteps; ++ks)
            mma_bf16_ss(tmem + (uint32_t)((i & 1) * NH), k_lo + (uint32_t)((ks >> 2) * (kPanel >> 4) + (ks & 3) * 2),
                        q_lo + (uint32_t)((ks >> 2) * (NH * 8) + (ks & 3) * 2), idesc_s, ks > 0 ? 1u : 0u);
          mma_commit(&s_ready[i & 1]);
          did = true;
        }
        if (did) {
          idle = 0;
        } else if (*reinterpret_cast<volatile int*>(&s_abort)) {
          ok = false;
        } else if (idle == 0) {
          idle = clock64();
        } else if (clock64() - idle > kWaitCycles) {
          s_abort = 1;
          atomicExch(&g_latent_fault, 1);
          ok = false;
        }
      }
      mma_commit(&finished);
      int no_abort = 0;
      mbar_wait(&finished, 0u, &no_abort, &g_latent_fault);
    }
  } else {
    {   // the heads' queries, K-major
      const int pieces = sh.panels * 8, live_pieces = a.dpad >> 3;
      const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + ((size_t)r * a.heads + h0) * a.dpad;
      for (int i = tid; i < NH * pieces; i += 128) {
        const int h = i / pieces, c = i - h * pieces;
        const bool live = h < nh && c < live_pieces;
        const int bytes = live ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(q_at + (uint32_t)((c >> 3) * NH * 128 + h * 128 + (((c & 7) ^ (h & 7)) << 4))),
                     "l"(q + (live ? (size_t)h * a.dpad + c * 8 : 0)), "r"(bytes)
                     : "memory");
      }
      asm volatile("cp.async.wait_all;" ::: "memory");
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      mbar_arrive(&q_full);
    }
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    const float scale = a.scale * kLog2E;
    constexpr int NB = NH / 8;           // blocks of eight heads
    // this lane's keys of a tile: 16 warp + lane / 4 and 8 on; heads 8 i + 2 (lane & 3) and the next
    const int key = warp * 16 + (lane >> 2), col = (lane & 3) * 2;
    float m = -INFINITY, l[NB][2];       // m: thread h of warp 0, head h;  l: these keys' share of the heads' sums
#pragma unroll
    for (int i = 0; i < NB; ++i) l[i][0] = l[i][1] = 0.f;
    bool ok = true;
    for (int t = 0; t < n; ++t) {
      ok = mbar_wait(&s_ready[t & 1], (uint32_t)(t >> 1) & 1u, &s_abort, &g_latent_fault);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) s_bad = 1;
      float s[NB][4];
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < NB; ++i) tmem_ld_tile(tmem + lanes + (uint32_t)((t & 1) * NH + i * 8), s[i]);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        const int p = begin + (t0 + t) * kKeys + key;
        const bool seen[2] = {p >= lo && p <= pos, p + 8 >= lo && p + 8 <= pos};
        float mx[NB][2];
#pragma unroll
        for (int i = 0; i < NB; ++i)
#pragma unroll
          for (int y = 0; y < 2; ++y) {
#pragma unroll
            for (int z = 0; z < 2; ++z) s[i][2 * z + y] = seen[z] ? s[i][2 * z + y] * scale : -INFINITY;
            mx[i][y] = fmaxf(s[i][y], s[i][2 + y]);
          }
#pragma unroll
        for (int o = 16; o > 2; o >>= 1)
#pragma unroll
          for (int i = 0; i < NB; ++i)
#pragma unroll
            for (int y = 0; y < 2; ++y) mx[i][y] = fmaxf(mx[i][y], __shfl_xor_sync(0xffffffffu, mx[i][y], o));
        if (lane < 4)
#pragma unroll
          for (int i = 0; i < NB; ++i) *reinterpret_cast<float2*>(&s_max[warp][i * 8 + col]) = make_float2(mx[i][0], mx[i][1]);
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      const bool bad = *reinterpret_cast<volatile int*>(&s_bad) != 0;   // the same for all four warps: written in front of this barrier only
      if (warp == 0) {
        bool grow = false;
        if (lane < NH) {
          const float mx = fmaxf(fmaxf(s_max[0][lane], s_max[1][lane]), fmaxf(s_max[2][lane], s_max[3][lane]));
          grow = mx > m + kGrow || (m == -INFINITY && mx != -INFINITY);
          const float m1 = grow ? fmaxf(m, mx) : m;
          s_alpha[lane] = m == -INFINITY ? 0.f : ex2(m - m1);
          s_ref[lane] = m1 == -INFINITY ? 0.f : m1;
          m = m1;
        }
        grow = __any_sync(0xffffffffu, grow);
        if (lane == 0) s_grown = grow ? 1 : 0;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (bad) {   // the abort word ends the other warps' waits
        ok = false;
        break;
      }
      if (s_grown) {
        if (t > 0) {
          mbar_wait(&pv_done[(t - 1) & 1], (uint32_t)((t - 1) >> 1) & 1u, &s_abort, &g_latent_fault);
          __syncwarp();
          tc_fence_after();
          for (int x = 0; x < 2 * sh.mtiles; ++x) {   // both pieces
            float o[NH];
            tmem_load<NH>(o_at + lanes + (uint32_t)(x * NH), o);
#pragma unroll
            for (int h = 0; h < NH; ++h) o[h] *= s_alpha[h];
#pragma unroll
            for (int h = 0; h < NH; h += 8) tmem_st8(o_at + lanes + (uint32_t)(x * NH + h), o + h);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
#pragma unroll
        for (int i = 0; i < NB; ++i)
#pragma unroll
          for (int y = 0; y < 2; ++y) l[i][y] *= s_alpha[i * 8 + col + y];
      }
      if (t > 1) mbar_wait(&pv_done[t & 1], (uint32_t)((t - 2) >> 1) & 1u, &s_abort, &g_latent_fault);   // the weights' place is free
      {
        // [key][head] -> [head][key]: this lane then has head 8 i + lane / 4, keys 2 (lane & 3) and the next of each block of eight
        unsigned char* p = smem + (p_at - k_at) + (size_t)(t & 1) * 2 * NH * 128 + (lane >> 2) * 128 + (lane & 3) * 4;
#pragma unroll
        for (int i = 0; i < NB; ++i) {
          const float2 ref = *reinterpret_cast<const float2*>(&s_ref[i * 8 + col]);
#pragma unroll
          for (int z = 0; z < 2; ++z) {
            const float w0 = ex2(s[i][2 * z] - ref.x), w1 = ex2(s[i][2 * z + 1] - ref.y);
            l[i][0] += w0;
            l[i][1] += w1;
            const uint32_t hi = pack2(w0, w1);
            const uint32_t rest = pack2(w0 - __uint_as_float(hi << 16), w1 - __uint_as_float(hi & 0xFFFF0000u));
            unsigned char* at = p + i * 1024 + (((warp * 2 + z) ^ (lane >> 2)) << 4);
            *reinterpret_cast<uint32_t*>(at) = transposed(hi);
            *reinterpret_cast<uint32_t*>(at + NH * 128) = transposed(rest);
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      }
      tc_fence_before();
      mbar_arrive(&p_ready[t & 1]);
    }
    if (ok && n > 0) mbar_wait(&pv_done[(n - 1) & 1], (uint32_t)((n - 1) >> 1) & 1u, &s_abort, &g_latent_fault);
    __syncwarp();
    tc_fence_after();
#pragma unroll
    for (int o = 16; o > 2; o >>= 1)
#pragma unroll
      for (int i = 0; i < NB; ++i)
#pragma unroll
        for (int y = 0; y < 2; ++y) l[i][y] += __shfl_xor_sync(0xffffffffu, l[i][y], o);
    if (lane < 4)
#pragma unroll
      for (int i = 0; i < NB; ++i) *reinterpret_cast<float2*>(&s_l[warp][i * 8 + col]) = make_float2(l[i][0], l[i][1]);
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const bool whole = sh.splits == 1;
    if (warp == 0 && lane < NH) {
      const float sum = (s_l[0][lane] + s_l[1][lane]) + (s_l[2][lane] + s_l[3][lane]);
      float f = sum > 0.f ? 1.f : 0.f;
      if (whole && sum > 0.f) {
        f = 1.f / sum;
        if (a.gate && lane < nh) f *= a.gate[(size_t)r * a.heads + h0 + lane];
      }
      s_alpha[lane] = f;
      if (!whole && lane < nh) a.part_ml[((size_t)split * a.r.rows + r) * a.heads + h0 + lane] = make_float2(m, sum);
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    float* parts = a.parts + (((size_t)split * a.r.rows + r) * a.heads + h0) * a.vdim + tid;
    for (int mt = 0; mt < sh.mtiles; ++mt) {
      const int c = mt * 128 + tid;
      float o[NH];
#pragma unroll
      for (int h = 0; h < NH; ++h) o[h] = 0.f;
      __syncwarp();
      if (n > 0) {
        float rest[NH];
        tmem_load<NH>(o_at + lanes + (uint32_t)(mt * 2 * NH), o);
        tmem_load<NH>(o_at + lanes + (uint32_t)(mt * 2 * NH + NH), rest);
#pragma unroll
        for (int h = 0; h < NH; ++h) o[h] = c < a.vdim && s_alpha[h] > 0.f ? (o[h] + rest[h]) * s_alpha[h] : 0.f;
      }
      if (!whole) {
        if (c < a.vdim) {
          float* p = parts + mt * 128;
#pragma unroll
          for (int h = 0; h < NH; ++h, p += a.vdim)
            if (h < nh) *p = o[h];
        }
      } else {
#pragma unroll
        for (int h = 0; h < NH; ++h)
          if (h < nh && c < flash_column_limit(a, h0 + h)) flash_store_column<true>(a, r, h0 + h, c, o[h]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
  }
}

bool latent_shape(const FlashArgs& a, int nh, LatentShape* sh, size_t* smem) {
  sh->panels = (a.dpad + 63) / 64;
  sh->mtiles = (a.vdim + 127) / 128;
  if ((2 * sh->mtiles + 2) * nh > kColumns) return false;
  sh->stage_bytes = (sh->panels > 2 * sh->mtiles ? sh->panels : 2 * sh->mtiles) * kPanel;
  // behind the tiles: the queries, two buffers of weights in two pieces
  const size_t rest = (size_t)sh->panels * nh * 128 + (size_t)4 * nh * 128 + 1024;
  const size_t fit = (224 * 1024 - rest) / sh->stage_bytes;
  if (rest > 224 * 1024 || fit < 2) return false;
  sh->stages = fit < kStagesMax ? (int)fit : kStagesMax;
  *smem = rest + (size_t)sh->stages * sh->stage_bytes;
  return true;
}

}  // namespace

int flash_latent_fault_flag() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_latent_fault, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

bool flash_latent_supported(const FlashArgs& a) {
  LatentShape sh;
  size_t smem = 0;
  return a.values_in_keys && !a.one_sequence && a.softcap == 0.f && a.slopes == nullptr && a.keep_first == 0 && a.geom.keep == 0 && a.geom.ring % kKeys == 0 &&
         a.cache_slots > 0 && (int64_t)a.cache_slots * a.geom.rows <= INT_MAX && latent_shape(a, a.heads <= 16 ? 16 : 32, &sh, &smem);
}

tb_status launch_flash_latent(const FlashArgs& a, cudaStream_t st, int* splits_out) {
  const int nh = a.heads <= 16 ? 16 : 32, groups = (a.heads + nh - 1) / nh;
  LatentShape sh;
  size_t smem = 0;
  CUtensorMap map;
  if (!latent_shape(a, nh, &sh, &smem)) return fail(TB_ERR_SHAPE, "latent attention: %d / %d elements", a.dpad, a.vdim);
  if (!tma_panel_map(&map, a.k_cache, a.dpad, (int64_t)a.cache_slots * a.geom.rows, a.dpad, kKeys))
    return fail(TB_ERR_CUDA, "latent attention: no tensor map of the cache");
  int64_t splits = (int64_t)sm_count() / ((int64_t)a.r.rows * groups);
  const int64_t tiles = (a.max_visible + 2 * kKeys - 2) / kKeys;
  if (splits > tiles) splits = tiles;
  if (splits > a.part_slots / ((int64_t)a.r.rows * a.heads)) splits = a.part_slots / ((int64_t)a.r.rows * a.heads);
  sh.splits = splits < 1 ? 1 : (int)splits;
  *splits_out = sh.splits;
  const dim3 grid((unsigned)sh.splits, (unsigned)groups, (unsigned)a.r.rows);
  return nh == 16 ? launch_kernel(flash_latent_kernel<16>, grid, dim3(kThreads), smem, st, a.pdl, 1, a, sh, map)
                  : launch_kernel(flash_latent_kernel<32>, grid, dim3(kThreads), smem, st, a.pdl, 1, a, sh, map);
}

}  // namespace tb

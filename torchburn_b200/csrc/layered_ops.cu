// Row kernels of the layered decoder, between the projections: residual + norms + the causal convolution
// in front of a sublayer (glue), query/key norm with the cache append (over the whole projection or per head),
// the latent's norm and rotation, PolyNorm and the squared relu.  All arithmetic is fp32; the results are
// written as the next projection's operand.
//
// A row is handled by a cluster of 1..8 CTAs (few rows: more CTAs, so that a decode row of several thousand
// features is not one SM's work); block sums meet through distributed shared memory and are added in rank
// order, so a result does not depend on timing.  The partial sums of a K-split projection are added here.
#include <cooperative_groups.h>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace tb {

namespace {

constexpr int kThreads = 256;

// Sum over the cluster of N values per thread.  `slot` alternates 0, 1, 0, ... from call to call: a CTA that
// has passed the barrier of call i has finished reading the slot of call i - 1.
template <int N>
struct ClusterSum {
  float part[N][kThreads / 32];
  float all[2][8][N];
};
template <int N>
__device__ __forceinline__ void cluster_sum(ClusterSum<N>& s, int slot, int csize, int crank, float (&v)[N]) {
#pragma unroll
  for (int i = 0; i < N; ++i)
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v[i] += __shfl_xor_sync(0xffffffffu, v[i], o);
  if ((threadIdx.x & 31) == 0)
#pragma unroll
    for (int i = 0; i < N; ++i) s.part[i][threadIdx.x >> 5] = v[i];
  __syncthreads();
  if (csize == 1) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < kThreads / 32; ++w) t += s.part[i][w];
      v[i] = t;
    }
    __syncthreads();   // `part` may be rewritten
    return;
  }
  cg::cluster_group cl = cg::this_cluster();
  if (threadIdx.x < (unsigned)csize) {
    ClusterSum<N>* peer = cl.map_shared_rank(&s, threadIdx.x);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < kThreads / 32; ++w) t += s.part[i][w];
      peer->all[slot][crank][i] = t;
    }
  }
  cl.sync();
#pragma unroll
  for (int i = 0; i < N; ++i) {
    float t = 0.f;
    for (int r = 0; r < csize; ++r) t += s.all[slot][r][i];
    v[i] = t;
  }
}

__device__ __forceinline__ float4 f4(float v) { return make_float4(v, v, v, v); }
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float dot4(float4 a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 scale4(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
constexpr int kMaxParts = 8;
__device__ __forceinline__ float4 sum_partials(const PartialSums& y, int row, int col) {
  const float* p = y.y + (size_t)row * y.ldy + col;
  float4 t[kMaxParts];   // every load in flight before the first sum
#pragma unroll
  for (int s = 0; s < kMaxParts; ++s)
    if (s < y.splits) t[s] = ld4(p + (size_t)s * y.split_stride);
  float4 v = t[0];
#pragma unroll
  for (int s = 1; s < kMaxParts; ++s)
    if (s < y.splits) v = add4(v, t[s]);
  return v;
}
// Four features of the embedding of token `tok` at position `pos`, from k on: the tile images of the tied output
// matrix, scaled, plus the position row.
__device__ __forceinline__ float4 embed4(const GlueArgs& a, int tok, int pos, int k) {
  const unsigned char* t = static_cast<const unsigned char*>(a.embed.img) + ((size_t)(tok >> 7) * (a.embed.kp >> 6) + (k >> 6)) * 16384 +
                           (size_t)(tok & 127) * 128 + ((((k >> 3) & 7) ^ (tok & 7)) << 4) + ((k & 7) << 1);
  const uint2 u = *reinterpret_cast<const uint2*>(t);
  float4 v = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
  v = scale4(v, a.embed_scale);
  if (a.pos_table) {
    const __nv_bfloat16* pr = a.pos_table + (size_t)pos * a.width;
    if (k < a.width) v.x += __bfloat162float(pr[k]);
    if (k + 1 < a.width) v.y += __bfloat162float(pr[k + 1]);
    if (k + 2 < a.width) v.z += __bfloat162float(pr[k + 2]);
    if (k + 3 < a.width) v.w += __bfloat162float(pr[k + 3]);
  }
  return v;
}
// Is row q of the step the position r - q in front of row r's, in the same sequence?
__device__ __forceinline__ bool same_run(const int32_t* slots, const int32_t* posv, int q, int r) {
  return q >= 0 && slots[q] == slots[r] && posv[q] >= 0 && posv[q] == posv[r] - (r - q);
}

// Many rows, first half of the glue: one CTA per row, x' and 1 / rms(x').
__global__ void __launch_bounds__(kThreads) residual_norm_kernel(const GlueArgs a, const int e4) {
  extern __shared__ float4 s_dyn[];   // [e4][kThreads]
  __shared__ ClusterSum<1> s_sum;
  const int tid = threadIdx.x, r = (int)blockIdx.x, xs4 = a.xs >> 2;
  grid_dep_launch();
  grid_dep_wait();
  const bool emb = a.embed.img != nullptr;
  int tok = 0, pos = 0;
  if (emb) {
    tok = a.r.tokens[r];
    pos = a.r.offsets[r];
    if (!(tok >= 0 && tok < a.vocab && pos >= 0 && pos < a.max_pos)) pos = -1;
    if (tid == 0) a.r.pos[r] = pos;
  }
  float inv = 1.f;
  float ss[1] = {0.f};
  for (int e = 0, i = tid; i < xs4; ++e, i += kThreads) {
    float4 v = f4(0.f);
    if (!emb) {
      v = sum_partials(a.y, r, i * 4);
      if (a.y_bias) v = add4(v, ld4(a.y_bias + i * 4));
    } else if (pos >= 0) {
      v = embed4(a, tok, pos, i * 4);
    }
    s_dyn[e * kThreads + tid] = v;
    ss[0] += dot4(v);
  }
  if (a.post_w) {
    cluster_sum<1>(s_sum, 0, 1, 0, ss);
    inv = 1.0f / sqrtf(ss[0] / (float)a.width + a.eps);
  }
  ss[0] = 0.f;
  for (int e = 0, i = tid; i < xs4; ++e, i += kThreads) {
    const float4 y = s_dyn[e * kThreads + tid];
    float4 v = emb ? f4(0.f) : ld4(a.x_in + (size_t)r * a.xs + i * 4);
    v = a.post_w ? fma4(scale4(y, inv), ld4(a.post_w + i * 4), v) : add4(v, y);
    ss[0] += dot4(v);
    *reinterpret_cast<float4*>(a.x_out + (size_t)r * a.xs + i * 4) = v;
    if (a.snapshot) *reinterpret_cast<float4*>(a.snapshot + (size_t)r * a.xs + i * 4) = v;
  }
  cluster_sum<1>(s_sum, 0, 1, 0, ss);
  if (tid == 0) a.rstd[r] = 1.0f / sqrtf(ss[0] / (float)a.width + a.eps);
}

// Second half: h = x' * rstd * pre_w, the convolution, the operand, the convolution's state.  grid (rows, columns / 1024)
template <bool BF16>
__global__ void __launch_bounds__(kThreads) norm_conv_kernel(const GlueArgs a) {
  const int r = a.row0 + (int)blockIdx.x, i = (int)blockIdx.y * kThreads + threadIdx.x;
  grid_dep_launch();
  grid_dep_wait();
  if (i >= (a.xs >> 2)) return;
  const int pos = a.r.pos[r];
  const float4 pw = ld4(a.pre_w + i * 4);
  auto input = [&](int q) { return mul4(scale4(ld4(a.x_out + (size_t)q * a.xs + i * 4), a.rstd[q]), pw); };
  const float4 h = input(r);
  if (a.write_state && pos >= 0)
    *reinterpret_cast<float4*>(a.conv_state + ((size_t)a.r.slots[r] * a.ring + (pos & (a.ring - 1))) * a.xs + i * 4) = h;
  const int orow = a.row_map != nullptr ? a.row_map[r] : r;
  if (a.out.data == nullptr || orow < 0) return;
  float4 o = h;
  if (a.conv_w != nullptr && pos >= 0) {
    for (int j = 0; j < a.taps && j <= pos; ++j) {
      float4 hp = h;
      if (j > 0) {
        if (same_run(a.r.slots, a.r.pos, r - j, r)) hp = input(r - j);
        else hp = ld4(a.conv_state + ((size_t)a.r.slots[r] * a.ring + ((pos - j) & (a.ring - 1))) * a.xs + i * 4);
      }
      o = fma4(ld4(a.conv_w + (size_t)(a.taps - 1 - j) * a.xs + i * 4), hp, o);
    }
  }
  if (pos < 0) o = f4(0.f);
  act_store4<BF16>(a.out, orow, i * 4, o);
}

// grid: (rows / rows_per * csize); rows_per consecutive rows per cluster, after up to taps - 1 rows of the same
// sequence in front of them whose convolution inputs are computed again.
template <bool BF16>
__global__ void __launch_bounds__(kThreads) glue_kernel(const GlueArgs a, const int rows_per, const int e4) {
  extern __shared__ float4 s_dyn[];        // [1 + taps][e4][kThreads]: x' of the row, then h of the last taps rows
  __shared__ ClusterSum<1> s_sum;
  const int tid = threadIdx.x;
  const int csize = (int)cg::this_cluster().num_blocks();
  const int crank = (int)cg::this_cluster().block_rank();
  const int xs4 = a.xs >> 2, lane4 = crank * kThreads + tid, step4 = csize * kThreads;
  const int r0 = a.row0 + ((int)blockIdx.x / csize) * rows_per;
  const int r1 = min(a.r.rows, r0 + rows_per);
  float4* s_x = s_dyn;
  float4* s_h = s_dyn + (size_t)e4 * kThreads;
  const int hist = e4 * kThreads;
  if (csize > 1) cg::this_cluster().sync();   // every CTA of the cluster runs before its shared memory is written
  grid_dep_launch();
  grid_dep_wait();
  const int taps = a.conv_w != nullptr ? a.taps : 1;
  const bool emb = a.embed.img != nullptr;
  int slot = 0;
  const int32_t* posv = emb ? a.r.offsets : a.r.pos;   // the embedding kernel is the one that writes r.pos

  for (int r = max(0, r0 - (taps - 1)); r < r1; ++r) {
    if (r < r0 && !same_run(a.r.slots, posv, r, r0)) continue;
    // ---- x' ----
    int tok = 0, pos = posv[r];
    bool live = pos >= 0;
    if (emb) {
      tok = a.r.tokens[r];
      live = tok >= 0 && tok < a.vocab && pos >= 0 && pos < a.max_pos;
      if (!live) pos = -1;
      if (r >= r0 && tid == 0 && crank == 0) a.r.pos[r] = pos;
    }
    float inv = 1.f;
    const bool source = emb || a.y.y != nullptr;
    if (source) {
      float ss[1] = {0.f};
      for (int e = 0, i = lane4; i < xs4; ++e, i += step4) {
        float4 v = f4(0.f);
        if (!emb) {
          v = sum_partials(a.y, r, i * 4);
          if (a.y_bias) v = add4(v, ld4(a.y_bias + i * 4));
        } else if (live) {
          v = embed4(a, tok, pos, i * 4);
        }
        s_x[e * kThreads + tid] = v;
        ss[0] += dot4(v);
      }
      if (a.post_w) {
        cluster_sum<1>(s_sum, slot, csize, crank, ss);
        slot ^= 1;
        inv = 1.0f / sqrtf(ss[0] / (float)a.width + a.eps);
      }
    }
    float ss[1] = {0.f};
    for (int e = 0, i = lane4; i < xs4; ++e, i += step4) {
      float4 v = emb ? f4(0.f) : ld4(a.x_in + (size_t)r * a.xs + i * 4);
      if (source) {
        const float4 y = s_x[e * kThreads + tid];
        v = a.post_w ? fma4(scale4(y, inv), ld4(a.post_w + i * 4), v) : add4(v, y);
      }
      s_x[e * kThreads + tid] = v;
      ss[0] += dot4(v);
      if (r >= r0 && a.x_out) *reinterpret_cast<float4*>(a.x_out + (size_t)r * a.xs + i * 4) = v;
      if (r >= r0 && a.snapshot) *reinterpret_cast<float4*>(a.snapshot + (size_t)r * a.xs + i * 4) = v;
    }
    // ---- h = norm(x') ----
    cluster_sum<1>(s_sum, slot, csize, crank, ss);
    slot ^= 1;
    inv = 1.0f / sqrtf(ss[0] / (float)a.width + a.eps);
    const int orow = (a.row_map != nullptr && r >= r0) ? a.row_map[r] : r;
    uint32_t in_step = 0;   // bit j: the input j positions back is a row of this step (else it is in the state)
    for (int j = 1; j < taps; ++j) in_step |= same_run(a.r.slots, posv, r - j, r) ? 1u << j : 0u;
    float4* h_cur = s_h + (size_t)(r % taps) * hist;
    for (int e = 0, i = lane4; i < xs4; ++e, i += step4) {
      const float4 h = mul4(scale4(s_x[e * kThreads + tid], inv), ld4(a.pre_w + i * 4));
      h_cur[e * kThreads + tid] = h;
      if (r < r0) continue;
      if (a.write_state && pos >= 0)
        *reinterpret_cast<float4*>(a.conv_state + ((size_t)a.r.slots[r] * a.ring + (pos & (a.ring - 1))) * a.xs + i * 4) = h;
      if (a.out.data == nullptr || orow < 0) continue;
      float4 o = h;
      if (a.conv_w != nullptr && pos >= 0) {
        for (int j = 0; j < taps && j <= pos; ++j) {   // tap taps - 1 - j meets the input j positions back
          float4 hp = h;
          if (j > 0) {
            if ((in_step >> j) & 1u) hp = s_h[(size_t)((r - j) % taps) * hist + e * kThreads + tid];
            else hp = ld4(a.conv_state + ((size_t)a.r.slots[r] * a.ring + ((pos - j) & (a.ring - 1))) * a.xs + i * 4);
          }
          o = fma4(ld4(a.conv_w + (size_t)(taps - 1 - j) * a.xs + i * 4), hp, o);
        }
      }
      if (pos < 0) o = f4(0.f);
      act_store4<BF16>(a.out, orow, i * 4, o);
    }
  }
}

// Many rows, x' = x + y without a norm of y and without a convolution: one CTA per row, everything in registers.
template <bool BF16, int E>
__global__ void __launch_bounds__(kThreads) glue_row_kernel(const GlueArgs a) {
  __shared__ ClusterSum<1> s_sum;
  const int tid = threadIdx.x, r = a.row0 + (int)blockIdx.x, xs4 = a.xs >> 2;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r], orow = a.row_map != nullptr ? a.row_map[r] : r;
  float4 v[E], y[E];
  float ss[1] = {0.f};
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = tid + e * kThreads;
    if (i >= xs4) continue;
    v[e] = ld4(a.x_in + (size_t)r * a.xs + i * 4);
    y[e] = sum_partials(a.y, r, i * 4);
  }
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = tid + e * kThreads;
    if (i >= xs4) continue;
    if (a.y_bias) y[e] = add4(y[e], ld4(a.y_bias + i * 4));
    v[e] = add4(v[e], y[e]);
    ss[0] += dot4(v[e]);
    if (a.x_out) *reinterpret_cast<float4*>(a.x_out + (size_t)r * a.xs + i * 4) = v[e];
    if (a.snapshot) *reinterpret_cast<float4*>(a.snapshot + (size_t)r * a.xs + i * 4) = v[e];
  }
  cluster_sum<1>(s_sum, 0, 1, 0, ss);
  if (a.out.data == nullptr || orow < 0) return;
  const float inv = 1.0f / sqrtf(ss[0] / (float)a.width + a.eps);
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = tid + e * kThreads;
    if (i < xs4) act_store4<BF16>(a.out, orow, i * 4, pos < 0 ? f4(0.f) : mul4(scale4(v[e], inv), ld4(a.pre_w + i * 4)));
  }
}

// Decode rows: every row its own sequence, four features per thread.  The same arithmetic as glue_kernel; the
// weights are read before the grid dependency wait, everything else as soon as its address is known.
constexpr int kStepTaps = 8;
template <bool BF16>
__global__ void __launch_bounds__(kThreads) glue_step_kernel(const GlueArgs a) {
  __shared__ ClusterSum<1> s_sum;
  const int tid = threadIdx.x;
  const int csize = (int)cg::this_cluster().num_blocks();
  const int crank = (int)cg::this_cluster().block_rank();
  const int r = a.row0 + (int)blockIdx.x / csize, i = crank * kThreads + tid;
  const bool in = i < (a.xs >> 2), emb = a.embed.img != nullptr;
  const int taps = a.conv_w != nullptr ? a.taps : 1;
  const float4 zero = f4(0.f);
  float4 pw = zero, ow = zero, bias = zero, cw[kStepTaps];
  if (in) {
    pw = ld4(a.pre_w + i * 4);
    if (a.post_w) ow = ld4(a.post_w + i * 4);
    if (!emb && a.y_bias) bias = ld4(a.y_bias + i * 4);
#pragma unroll
    for (int j = 0; j < kStepTaps; ++j)
      if (a.conv_w != nullptr && j < taps) cw[j] = ld4(a.conv_w + (size_t)(taps - 1 - j) * a.xs + i * 4);
  }
  if (csize > 1) cg::this_cluster().sync();
  grid_dep_launch();
  grid_dep_wait();
  int tok = 0, pos = emb ? a.r.offsets[r] : a.r.pos[r];
  if (emb) {
    tok = a.r.tokens[r];
    if (!(tok >= 0 && tok < a.vocab && pos >= 0 && pos < a.max_pos)) pos = -1;
    if (tid == 0 && crank == 0) a.r.pos[r] = pos;
  }
  float4 v = zero, x = zero, prev[kStepTaps];
  if (in && !emb) {
    x = ld4(a.x_in + (size_t)r * a.xs + i * 4);
    v = add4(sum_partials(a.y, r, i * 4), bias);
  }
  float* state = a.conv_w != nullptr ? a.conv_state + (size_t)a.r.slots[r] * a.ring * a.xs + i * 4 : nullptr;
  if (in && a.conv_w != nullptr) {
#pragma unroll
    for (int j = 1; j < kStepTaps; ++j)
      if (j < taps && j <= pos) prev[j] = ld4(state + (size_t)((pos - j) & (a.ring - 1)) * a.xs);
  }
  float ss[1];
  if (emb && in && pos >= 0) v = embed4(a, tok, pos, i * 4);
  if (a.post_w) {
    ss[0] = dot4(v);
    cluster_sum<1>(s_sum, 0, csize, crank, ss);
    v = fma4(scale4(v, 1.0f / sqrtf(ss[0] / (float)a.width + a.eps)), ow, x);
  } else {
    v = add4(x, v);
  }
  ss[0] = dot4(v);
  cluster_sum<1>(s_sum, 1, csize, crank, ss);
  if (!in) return;
  if (a.x_out) *reinterpret_cast<float4*>(a.x_out + (size_t)r * a.xs + i * 4) = v;
  if (a.snapshot) *reinterpret_cast<float4*>(a.snapshot + (size_t)r * a.xs + i * 4) = v;
  const float4 h = mul4(scale4(v, 1.0f / sqrtf(ss[0] / (float)a.width + a.eps)), pw);
  if (a.write_state && pos >= 0) *reinterpret_cast<float4*>(state + (size_t)(pos & (a.ring - 1)) * a.xs) = h;
  const int orow = a.row_map != nullptr ? a.row_map[r] : r;
  if (a.out.data == nullptr || orow < 0) return;
  float4 o = h;
  if (a.conv_w != nullptr) {
#pragma unroll
    for (int j = 0; j < kStepTaps; ++j)
      if (j < taps && j <= pos) o = fma4(cw[j], j == 0 ? h : prev[j], o);
  }
  if (pos < 0) o = zero;
  act_store4<BF16>(a.out, orow, i * 4, o);
}

// Query/key norm over the whole projection, biases, heads split and padded, k and v into the cache.
template <typename T>
__global__ void __launch_bounds__(kThreads) qkv_prep_kernel(const QkvPrepArgs a, const int e4) {
  extern __shared__ float4 s_val[];   // [e4][kThreads]: this thread's pieces of the row, summed
  __shared__ ClusterSum<2> s_sum;
  const int tid = threadIdx.x;
  const int csize = (int)cg::this_cluster().num_blocks();
  const int crank = (int)cg::this_cluster().block_rank();
  const int r = (int)blockIdx.x / csize;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
  const int cols4 = (a.v_off + nv + 3) >> 2, k4 = a.k_off >> 2, v4 = a.v_off >> 2;
  const int first = crank * kThreads + tid, step = csize * kThreads;
  if (csize > 1) cg::this_cluster().sync();
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  float ss[2] = {0.f, 0.f};
  for (int e = 0, i = first; i < cols4; ++e, i += step) {   // padded columns are zero
    float4 v = sum_partials(a.y, r, i * 4);
    if (a.bias) v = add4(v, ld4(a.bias + i * 4));
    s_val[e * kThreads + tid] = v;
    if (i < k4) ss[0] += dot4(v);
    else if (i < v4) ss[1] += dot4(v);
  }
  cluster_sum<2>(s_sum, 0, csize, crank, ss);
  const float iq = a.q_norm ? 1.0f / sqrtf(ss[0] / (float)nq + a.eps) : 1.f;
  const float ik = a.k_norm ? 1.0f / sqrtf(ss[1] / (float)nk + a.eps) : 1.f;
  const size_t crow = pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows + a.geom.row_of(pos);
  T* kc = static_cast<T*>(a.k_cache) + crow * (size_t)(a.kv_heads * a.dpad);
  T* vc = static_cast<T*>(a.v_cache) + crow * (size_t)(a.kv_heads * a.vpad);
  for (int e = 0, i = first; i < cols4; ++e, i += step) {
    const float4 v4v = s_val[e * kThreads + tid];
    const float v[4] = {v4v.x, v4v.y, v4v.z, v4v.w};
    // segment of this piece: segments start at multiples of 4
    const int seg = i < k4 ? 0 : (i < v4 ? 1 : 2);
    const int base = i * 4 - (seg == 0 ? 0 : (seg == 1 ? a.k_off : a.v_off));
    const int n = seg == 0 ? nq : (seg == 1 ? nk : nv), d = seg == 2 ? a.vdim : a.dim, dp = seg == 2 ? a.vpad : a.dpad;
    int head = base / d, c = base - head * d;
#pragma unroll
    for (int j = 0; j < 4; ++j, ++c) {
      if (base + j >= n) break;
      if (c == d) { c = 0; ++head; }
      const size_t o = (size_t)head * dp + c;
      if (seg == 0) {
        const float q = v[j] * iq * (a.q_norm ? a.q_norm[base + j] : 1.f);
        if (a.q) a.q[(size_t)r * a.heads * a.dpad + o] = q;
        if (a.q16) a.q16[(size_t)r * a.heads * a.dpad + o] = __float2bfloat16_rn(q);
      } else if (pos >= 0) {
        if (seg == 1) kc[o] = (T)(v[j] * ik * (a.k_norm ? a.k_norm[base + j] : 1.f));
        else vc[o] = (T)v[j];
      }
    }
  }
}

// One column of a projection: its partial sums in order.
__device__ __forceinline__ float sum_column(const PartialSums& y, int row, int col) {
  const float* p = y.y + (size_t)row * y.ldy + col;
  float t[kMaxParts];
#pragma unroll
  for (int s = 0; s < kMaxParts; ++s)
    if (s < y.splits) t[s] = p[(size_t)s * y.split_stride];
  float v = t[0];
#pragma unroll
  for (int s = 1; s < kMaxParts; ++s)
    if (s < y.splits) v += t[s];
  return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Per head: a warp takes one head of q, k or v through its norm (or the value mixing) to where it goes; one more
// warp per 32 heads does the gates.  grid (warps of a row / 8, rows)
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// V4: sizes are multiples of four, a lane takes four columns at a time; else one.
template <typename T, bool V4>
__global__ void __launch_bounds__(kThreads) heads_prep_kernel(const HeadsPrepArgs a) {
  [[maybe_unused]] constexpr int KEEP = 8;                  // values a lane keeps between the norm's two passes
  const int lane = threadIdx.x & 31, r = (int)blockIdx.y;
  int u = (int)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  const size_t crow = pos < 0 ? 0 : (size_t)a.r.slots[r] * a.geom.rows + a.geom.row_of(pos);
  if (u < a.heads + a.kv_heads) {
    const bool is_q = u < a.heads;
    const int h = is_q ? u : u - a.heads, col = (is_q ? a.q_off : a.k_off) + h * a.dim;
    float v[KEEP], ss = 0.f;
    float4 w4[2];
    if constexpr (V4) {
      for (int c = lane * 4, e = 0; c < a.dim; c += 128, ++e) {
        const float4 x = sum_partials(a.y, r, col + c);
        if (e == 0) w4[0] = x;
        else if (e == 1) w4[1] = x;
        ss += dot4(x);
      }
    } else {
#pragma unroll
      for (int j = 0; j < KEEP; ++j)
        if (lane + 32 * j < a.dim) {
          v[j] = sum_column(a.y, r, col + lane + 32 * j);
          ss = fmaf(v[j], v[j], ss);
        }
      for (int c = lane + 32 * KEEP; c < a.dim; c += 32) {
        const float x = sum_column(a.y, r, col + c);
        ss = fmaf(x, x, ss);
      }
    }
    const float inv = a.unit_norm ? 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps) : 1.f;
    T* dst = is_q ? static_cast<T*>(a.q) + ((size_t)r * a.heads + h) * a.dpad
                  : static_cast<T*>(a.k_cache) + crow * (size_t)(a.kv_heads * a.dpad) + h * a.dpad;
    if (!is_q && pos < 0) return;
    if constexpr (V4) {
      for (int c = lane * 4, e = 0; c < a.dim; c += 128, ++e) store4(dst + c, scale4(e == 0 ? w4[0] : (e == 1 ? w4[1] : sum_partials(a.y, r, col + c)), inv));
    } else {
#pragma unroll
      for (int j = 0; j < KEEP; ++j)
        if (lane + 32 * j < a.dim) dst[lane + 32 * j] = (T)(v[j] * inv);
      for (int c = lane + 32 * KEEP; c < a.dim; c += 32) dst[c] = (T)(sum_column(a.y, r, col + c) * inv);
    }
    return;
  }
  u -= a.heads + a.kv_heads;
  if (u < a.kv_heads) {
    T* dst = static_cast<T*>(a.v_cache) + crow * (size_t)(a.kv_heads * a.vpad) + u * a.vpad;
    float* first = a.v_first ? a.v_first + (size_t)r * a.kv_heads * a.vdim + u * a.vdim : nullptr;
    if constexpr (V4) {
      for (int c = lane * 4; c < a.vdim; c += 128) {
        float4 v = sum_partials(a.y, r, a.v_off + u * a.vdim + c);
        if (first && a.keep_first_values) store4(first + c, v);
        else if (first) v = fma4(f4(a.mix), ld4(first + c), scale4(v, 1.f - a.mix));
        if (pos >= 0) store4(dst + c, v);
      }
    } else {
      for (int c = lane; c < a.vdim; c += 32) {
        float v = sum_column(a.y, r, a.v_off + u * a.vdim + c);
        if (first && a.keep_first_values) first[c] = v;
        else if (first) v = fmaf(a.mix, first[c], (1.f - a.mix) * v);
        if (pos >= 0) dst[c] = (T)v;
      }
    }
    return;
  }
  const int g = (u - a.kv_heads) * 32 + lane;
  if (a.gate && g < a.heads) a.gate[(size_t)r * a.heads + g] = 1.0f / (1.0f + expf(-sum_column(a.y, r, a.g_off + g)));
}

// Rotation of dimensions 2i, 2i + 1 below `dims` at position pos; the others pass.
__device__ __forceinline__ float rotated(const float2* table, int dims, int pos, int c, float own, float other) {
  if (c >= dims || pos < 0) return own;
  const float2 cs = table[(size_t)pos * (dims >> 1) + (c >> 1)];
  return (c & 1) ? fmaf(own, cs.x, other * cs.y) : fmaf(own, cs.x, -other * cs.y);
}

// The latents of a row.  grid (2, rows): block 0 the query latent, normed, as the next product's operand; block 1
// the key/value latent, normed, and the shared rotated key part, into the cache.
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_prep_kernel(const LatentPrepArgs a) {
  extern __shared__ float s_lat[];
  __shared__ ClusterSum<1> s_sum;
  const int tid = threadIdx.x, r = (int)blockIdx.y;
  const bool is_q = blockIdx.x == 0;
  const int n = is_q ? a.q_rank : a.kv_rank, off = is_q ? 0 : a.kv_off;
  grid_dep_launch();
  grid_dep_wait();
  const int pos = a.r.pos[r];
  float ss[1] = {0.f};
  for (int c = tid; c < n; c += kThreads) {
    const float v = sum_column(a.y, r, off + c);
    s_lat[c] = v;
    ss[0] = fmaf(v, v, ss[0]);
  }
  cluster_sum<1>(s_sum, 0, 1, 0, ss);
  const float inv = 1.0f / sqrtf(ss[0] / (float)n + a.eps);
  if (is_q) {
    for (int c = tid; c < a.out.kp; c += kThreads) act_store1<sizeof(T) == 2>(a.out, r, c, c < n ? s_lat[c] * inv * a.q_norm[c] : 0.f);
    return;
  }
  if (pos < 0) return;
  T* row = static_cast<T*>(a.cache) + ((size_t)a.r.slots[r] * a.geom.rows + a.geom.row_of(pos)) * (size_t)a.dpad;
  for (int c = tid; c < n; c += kThreads) row[c] = (T)(s_lat[c] * inv * a.kv_norm[c]);
  for (int c = tid; c < a.rot_dim; c += kThreads) {
    const float own = sum_column(a.y, r, off + n + c), other = c < a.rot_dims ? sum_column(a.y, r, off + n + (c ^ 1)) : 0.f;
    row[n + c] = (T)rotated(a.table, a.rot_dims, pos, c, own, other);
  }
}

// The heads' queries after the up-projection: the unrotated part as the operand of the product with the head's
// key matrix, the rotated part behind the place of that product in the query.  Warp per head, grid (heads / 8, rows)
template <typename T, bool V4>
__global__ void __launch_bounds__(kThreads) latent_query_kernel(const LatentQueryArgs a) {
  const int lane = threadIdx.x & 31, r = (int)blockIdx.y, h = (int)blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  grid_dep_launch();
  grid_dep_wait();
  if (h >= a.heads) return;
  const int pos = a.r.pos[r], col = h * (a.dim + a.rot_dim);
  T* q = static_cast<T*>(a.q) + ((size_t)r * a.heads + h) * a.dpad;
  if constexpr (V4) {
    ActOperand out = a.out;
    if (out.data) out.data = static_cast<unsigned char*>(out.data) + (size_t)h * out.mp * out.kp * sizeof(T);
    const int n = out.data ? out.kp : a.dim;
    for (int c = lane * 4; c < n; c += 128) {
      const float4 v = c < a.dim ? sum_partials(a.y, r, col + c) : f4(0.f);
      if (out.data) act_store4<sizeof(T) == 2>(out, r, c, v);
      else store4(q + c, v);
    }
    q += a.rot_at;
    for (int c = lane * 4; c < a.rot_dim; c += 128) {
      const float4 v = sum_partials(a.y, r, col + a.dim + c);
      store4(q + c, make_float4(rotated(a.table, a.rot_dims, pos, c, v.x, v.y), rotated(a.table, a.rot_dims, pos, c + 1, v.y, v.x),
                                rotated(a.table, a.rot_dims, pos, c + 2, v.z, v.w), rotated(a.table, a.rot_dims, pos, c + 3, v.w, v.z)));
    }
  } else {
    if (a.out.data) {
      ActOperand out = a.out;
      out.data = static_cast<unsigned char*>(out.data) + (size_t)h * out.mp * out.kp * sizeof(T);
      for (int c = lane; c < out.kp; c += 32) act_store1<sizeof(T) == 2>(out, r, c, c < a.dim ? sum_column(a.y, r, col + c) : 0.f);
    } else {
      for (int c = lane; c < a.dim; c += 32) q[c] = (T)sum_column(a.y, r, col + c);
    }
    q += a.rot_at;
    for (int c = lane; c < a.rot_dim; c += 32) {
      const float own = sum_column(a.y, r, col + a.dim + c), other = c < a.rot_dims ? sum_column(a.y, r, col + a.dim + (c ^ 1)) : 0.f;
      q[c] = (T)rotated(a.table, a.rot_dims, pos, c, own, other);
    }
  }
}

// grid (positions, pieces / 256)
__global__ void __launch_bounds__(kThreads) latent_rows_kernel(const LatentRowsArgs a) {
  const int c = (int)blockIdx.y * kThreads + threadIdx.x, i = (int)blockIdx.x;
  grid_dep_launch();
  grid_dep_wait();
  if (c >= a.out.kp >> 3) return;
  const __nv_bfloat16* row = static_cast<const __nv_bfloat16*>(a.cache) + ((size_t)a.r.slots[0] * a.geom.rows + a.geom.row_of(a.lo + i)) * (size_t)a.dpad;
  const uint4 v = c * 8 < a.kv_rank ? *reinterpret_cast<const uint4*>(row + c * 8) : make_uint4(0u, 0u, 0u, 0u);
  *reinterpret_cast<uint4*>(static_cast<unsigned char*>(a.out.data) + image_offset(a.out.mp, i, c * 8)) = v;
}

// grid (columns / 1024, rows)
template <bool BF16>
__global__ void __launch_bounds__(kThreads) relu2_kernel(const PartialSums z, const ActOperand out) {
  const int k = ((int)blockIdx.x * kThreads + threadIdx.x) * 4, r = (int)blockIdx.y;
  grid_dep_launch();
  grid_dep_wait();
  if (k >= out.kp) return;
  float4 v = sum_partials(z, r, k);
  v = make_float4(fmaxf(v.x, 0.f), fmaxf(v.y, 0.f), fmaxf(v.z, 0.f), fmaxf(v.w, 0.f));
  act_store4<BF16>(out, r, k, mul4(v, v));
}

// Angles in fp64, so that a far position turns by its angle and not by a rounded one.
__global__ void __launch_bounds__(kThreads) rotation_table_kernel(float2* table, int64_t n, int half, double base) {
  const int64_t i = (int64_t)blockIdx.x * kThreads + threadIdx.x;
  if (i >= n) return;
  double sn, cs;
  sincos((double)(i / half) * pow(base, -(double)(i % half) / (double)half), &sn, &cs);
  table[i] = make_float2((float)cs, (float)sn);
}

template <bool BF16>
__global__ void __launch_bounds__(kThreads) poly_norm_kernel(const PolyNormArgs a, const int e4) {
  extern __shared__ float4 s_z[];   // [e4][kThreads]
  __shared__ ClusterSum<3> s_sum;
  const int tid = threadIdx.x;
  const int csize = (int)cg::this_cluster().num_blocks();
  const int crank = (int)cg::this_cluster().block_rank();
  const int r = (int)blockIdx.x / csize;
  const int k4 = a.out.kp >> 2, lane4 = crank * kThreads + tid, step4 = csize * kThreads;
  if (csize > 1) cg::this_cluster().sync();
  grid_dep_launch();
  grid_dep_wait();
  float ss[3] = {0.f, 0.f, 0.f};
  auto take = [&](int e, float4 z) {
    s_z[e * kThreads + tid] = z;
    const float4 z2 = mul4(z, z), z3 = mul4(z2, z);
    ss[0] += dot4(z);
    ss[1] += dot4(z2);
    ss[2] += dot4(z3);
  };
  if (a.z.splits == 1) {   // whole sums: several pieces in flight per thread
    const float* z = a.z.y + (size_t)r * a.z.ldy;
    int e = 0, i = lane4;
    for (; i + 3 * step4 < k4; e += 4, i += 4 * step4) {
      const float4 z0 = ld4(z + i * 4), z1 = ld4(z + (i + step4) * 4), z2 = ld4(z + (i + 2 * step4) * 4), z3 = ld4(z + (i + 3 * step4) * 4);
      take(e, z0);
      take(e + 1, z1);
      take(e + 2, z2);
      take(e + 3, z3);
    }
    for (; i < k4; ++e, i += step4) take(e, ld4(z + i * 4));
  } else {
    for (int e = 0, i = lane4; i < k4; ++e, i += step4) take(e, sum_partials(a.z, r, i * 4));
  }
  cluster_sum<3>(s_sum, 0, csize, crank, ss);
  const float n = (float)a.width;
  const float c1 = a.coef[0] / sqrtf(ss[0] / n + a.eps), c2 = a.coef[1] / sqrtf(ss[1] / n + a.eps), c3 = a.coef[2] / sqrtf(ss[2] / n + a.eps);
  const float c0 = a.coef[3];
  auto f = [&](float z, int k) { return k < a.width ? fmaf(z, fmaf(z, fmaf(z, c3, c2), c1), c0) : 0.f; };
  for (int e = 0, i = lane4; i < k4; ++e, i += step4) {
    const float4 z = s_z[e * kThreads + tid];
    const int k = i * 4;
    act_store4<BF16>(a.out, r, k, make_float4(f(z.x, k), f(z.y, k + 1), f(z.z, k + 2), f(z.w, k + 3)));
  }
}

// CTAs per row: enough to spread a few rows over the SMs, never more than there are 4-element pieces for.
int row_cluster(int rows, int64_t n4) {
  int c = 1;
  while (c < 8 && (int64_t)c * kThreads < n4 && rows * c * 2 <= sm_count()) c *= 2;
  return c;
}

}  // namespace

tb_status launch_glue(Precision p, const GlueArgs& a, cudaStream_t st) {
  const int n = a.r.rows - a.row0;
  if (n < 1) return TB_OK;
  if (a.rstd != nullptr) {   // many rows: two kernels, nothing computed twice
    const int e4 = (a.xs / 4 + kThreads - 1) / kThreads;
    if (a.taps > 32 || e4 > 50) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: hidden size %d with %d taps", a.width, a.taps);
    if (a.row0 == 0)
      TB_TRY(launch_kernel(residual_norm_kernel, dim3((unsigned)n), dim3(kThreads), (size_t)e4 * kThreads * sizeof(float4), st, a.pdl, 1, a, e4));
    const dim3 grid((unsigned)n, (unsigned)e4);
    return p == Precision::kBf16 ? launch_kernel(norm_conv_kernel<true>, grid, dim3(kThreads), 0, st, a.pdl, 1, a)
                                 : launch_kernel(norm_conv_kernel<false>, grid, dim3(kThreads), 0, st, a.pdl, 1, a);
  }
  const int c = row_cluster(n, a.xs / 4);
  int per = 1;
  if (c == 1 && a.conv_w)
    while (per < 4 && n / (per * 2) >= sm_count()) per *= 2;   // fewer rows computed again in front of each block
  const int e4 = (a.xs / 4 + c * kThreads - 1) / (c * kThreads);
  const int taps = a.conv_w ? a.taps : 1;
  const size_t smem = (size_t)(1 + taps) * e4 * kThreads * sizeof(float4);
  if (!a.neighbours && e4 == 1 && per == 1 && taps <= kStepTaps && (a.embed.img != nullptr || a.y.y != nullptr)) {
    const dim3 grid((unsigned)(n * c));
    return p == Precision::kBf16 ? launch_kernel(glue_step_kernel<true>, grid, dim3(kThreads), 0, st, a.pdl, c, a)
                                 : launch_kernel(glue_step_kernel<false>, grid, dim3(kThreads), 0, st, a.pdl, c, a);
  }
  if (c == 1 && !a.conv_w && !a.post_w && !a.embed.img && a.y.y != nullptr && e4 <= 4) {
    using Kernel = void (*)(GlueArgs);
    static const Kernel kernels[2][4] = {{glue_row_kernel<true, 1>, glue_row_kernel<true, 2>, glue_row_kernel<true, 3>, glue_row_kernel<true, 4>},
                                         {glue_row_kernel<false, 1>, glue_row_kernel<false, 2>, glue_row_kernel<false, 3>, glue_row_kernel<false, 4>}};
    return launch_kernel(kernels[p == Precision::kF32][e4 - 1], dim3((unsigned)n), dim3(kThreads), 0, st, a.pdl, 1, a);
  }
  if (smem > 200 * 1024 || taps > 32) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: hidden size %d with %d taps", a.width, a.taps);
  const dim3 grid((unsigned)((n + per - 1) / per * c));
  if (p == Precision::kBf16) return launch_kernel(glue_kernel<true>, grid, dim3(kThreads), smem, st, a.pdl, c, a, per, e4);
  return launch_kernel(glue_kernel<false>, grid, dim3(kThreads), smem, st, a.pdl, c, a, per, e4);
}

tb_status launch_qkv_prep(Precision p, const QkvPrepArgs& a, cudaStream_t st) {
  const int cols4 = (a.v_off + a.kv_heads * a.vdim + 3) / 4;
  const int c = row_cluster(a.r.rows, cols4);
  const int e4 = (cols4 + c * kThreads - 1) / (c * kThreads);
  const size_t smem = (size_t)e4 * kThreads * sizeof(float4);
  if (smem > 200 * 1024) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: %d query and %d key heads", a.heads, a.kv_heads);
  const dim3 grid((unsigned)(a.r.rows * c));
  if (p == Precision::kBf16) return launch_kernel(qkv_prep_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, st, a.pdl, c, a, e4);
  return launch_kernel(qkv_prep_kernel<float>, grid, dim3(kThreads), smem, st, a.pdl, c, a, e4);
}

tb_status launch_heads_prep(Precision p, const HeadsPrepArgs& a, cudaStream_t st) {
  const int warps = a.heads + 2 * a.kv_heads + (a.gate ? (a.heads + 31) / 32 : 0);
  const dim3 grid((unsigned)((warps + kThreads / 32 - 1) / (kThreads / 32)), (unsigned)a.r.rows);
  using Kernel = void (*)(HeadsPrepArgs);
  static const Kernel kernels[2][2] = {{heads_prep_kernel<__nv_bfloat16, false>, heads_prep_kernel<__nv_bfloat16, true>},
                                       {heads_prep_kernel<float, false>, heads_prep_kernel<float, true>}};
  return launch_kernel(kernels[p == Precision::kF32][a.dim % 4 == 0 && a.vdim % 4 == 0], grid, dim3(kThreads), 0, st, a.pdl, 1, a);
}

tb_status launch_latent_prep(Precision p, const LatentPrepArgs& a, cudaStream_t st) {
  const size_t smem = (size_t)(a.q_rank > a.kv_rank ? a.q_rank : a.kv_rank) * sizeof(float);
  if (smem > 200 * 1024) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: latents of %d and %d", a.q_rank, a.kv_rank);
  const dim3 grid(2, (unsigned)a.r.rows);
  return p == Precision::kBf16 ? launch_kernel(latent_prep_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, st, a.pdl, 1, a)
                               : launch_kernel(latent_prep_kernel<float>, grid, dim3(kThreads), smem, st, a.pdl, 1, a);
}

tb_status launch_latent_query(Precision p, const LatentQueryArgs& a, cudaStream_t st) {
  const dim3 grid((unsigned)((a.heads + kThreads / 32 - 1) / (kThreads / 32)), (unsigned)a.r.rows);
  using Kernel = void (*)(LatentQueryArgs);
  static const Kernel kernels[2][2] = {{latent_query_kernel<__nv_bfloat16, false>, latent_query_kernel<__nv_bfloat16, true>},
                                       {latent_query_kernel<float, false>, latent_query_kernel<float, true>}};
  const bool v4 = a.dim % 4 == 0 && a.rot_dim % 4 == 0 && a.rot_at % 4 == 0;
  return launch_kernel(kernels[p == Precision::kF32][v4], grid, dim3(kThreads), 0, st, a.pdl, 1, a);
}

tb_status launch_latent_rows(const LatentRowsArgs& a, cudaStream_t st) {
  const int pieces = a.out.kp >> 3, threads = pieces < kThreads ? (pieces + 31) / 32 * 32 : kThreads;
  return launch_kernel(latent_rows_kernel, dim3((unsigned)a.n, (unsigned)((pieces + kThreads - 1) / kThreads)), dim3((unsigned)threads), 0, st, a.pdl, 1, a);
}

tb_status launch_relu2(Precision p, int rows, const PartialSums& z, const ActOperand& out, bool pdl, cudaStream_t st) {
  const dim3 grid((unsigned)((out.kp / 4 + kThreads - 1) / kThreads), (unsigned)rows);
  return p == Precision::kBf16 ? launch_kernel(relu2_kernel<true>, grid, dim3(kThreads), 0, st, pdl, 1, z, out)
                               : launch_kernel(relu2_kernel<false>, grid, dim3(kThreads), 0, st, pdl, 1, z, out);
}

tb_status fill_rotation_table(float2* table, int64_t positions, int dims, double base) {
  const int64_t n = positions * (dims / 2);
  if (n == 0) return TB_OK;
  rotation_table_kernel<<<(unsigned)((n + kThreads - 1) / kThreads), kThreads>>>(table, n, dims / 2, base);
  TB_CUDA_TRY(cudaGetLastError());
  return TB_OK;
}

tb_status launch_poly_norm(Precision p, const PolyNormArgs& a, cudaStream_t st) {
  const int c = row_cluster(a.rows, a.out.kp / 4);
  const int e4 = (a.out.kp / 4 + c * kThreads - 1) / (c * kThreads);
  const size_t smem = (size_t)e4 * kThreads * sizeof(float4);
  if (smem > 200 * 1024) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: feed-forward width %d", a.width);
  const dim3 grid((unsigned)(a.rows * c));
  if (p == Precision::kBf16) return launch_kernel(poly_norm_kernel<true>, grid, dim3(kThreads), smem, st, a.pdl, c, a, e4);
  return launch_kernel(poly_norm_kernel<false>, grid, dim3(kThreads), smem, st, a.pdl, c, a, e4);
}

}  // namespace tb

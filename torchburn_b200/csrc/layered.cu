// The layered decoder: a stack of sublayers (mixer, optional feed-forward), each
//   x <- x + [norm_after] f(h + conv(h)),  h = norm_before(x)
// with its constants and sizes taken per layer from the caller.  Layers may share weights (weights_of); each
// run of a layer has its own cache and convolution states.
//
// One step is a chain of kernels per layer, by mixer
//   glue (residual, norms, convolution) -> QKV product -> query/key norm + cache append -> scores -> mix ->
//   output product -> glue -> up product -> PolyNorm -> down product                     (heads mixed by talk)
//   glue -> QKV (+ gate) product -> per-head norm, value mixing, cache append -> flash attention (-> merge) -> ...
//   glue -> latent product -> latent norms, rotation, cache append -> query product -> rotation -> key product per
//   head -> flash attention over the latents (-> merge) -> value product per head -> ...
//   (long portions: the latents of the sequence -> all heads' keys and values -> flash attention -> ...)
// and the final norm with the output product for the rows whose logits are wanted.  Every buffer between
// two kernels is written by exactly one of them and read by the next, so one buffer of partial sums and one
// operand buffer per kind serve the whole stack; the residual stream alternates between two buffers because
// the convolution recomputes its neighbours' rows.
//
// State of a sequence: per layer the rows of K and V, or of the latents (a ring behind a window or inside chunks:
// that many + a portion's rows + room to go back; the kept first positions have rows of their own) and per
// sublayer the last inputs of the convolution, by position in a ring.
#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "layered.cuh"
#include "window_attention.cuh"

namespace tb {

namespace {

constexpr int kHistory = 128;      // positions a sequence can always be taken back
constexpr int kMaxSplits = 8;
constexpr size_t kScoreBudget = 1024u << 20;
constexpr int kManyRows = 64;       // from here on the glue with a convolution is two kernels
constexpr int kExpandRows = 64;     // portions from here on write out the keys and values of latents
constexpr size_t kExpandBudget = (size_t)4096 << 20;
constexpr double kLaunchStages = 16.0;  // stages of a product's K loop that a kernel of its own costs

struct LayerWeights {
  bool latent = false;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dpad = 0, vpad = 0;
  int q_off = 0, k_off = 0, v_off = 0;
  int64_t qkv_cols = 0;
  int64_t ff = 0;
  float act[4] = {0, 0, 0, 0};
  DenseWeight qkv, o, up, down;    // qkv: [q | k | v | gates], or of a latent layer [query latent | key/value latent, rotated key]
  int g_off = 0;
  bool gate = false;
  float vmix = 0.f;
  int q_rank = 0, kv_rank = 0, rot_dim = 0;
  DenseWeight uq, uk, uv;            // uk: per head [kv_rank, dim], uv: per head [vdim, kv_rank]
  DenseWeight ukv;                   // [all heads' keys | all heads' values, kv_rank], where portions write them out
  int xpad = 0;                      // padded size of a written-out key
  float *dq_norm = nullptr, *dkv_norm = nullptr;
  float *qkv_b = nullptr, *q_norm = nullptr, *k_norm = nullptr, *talk = nullptr, *o_b = nullptr;
  float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
  float *conv1 = nullptr, *conv2 = nullptr;
};

struct LayerRun {
  int weights = 0;                 // index of the layer that owns the weights
  float scale = 1.f;
  int window = 0, keep_first = 0, chunk = 0;
  float softcap = 0.f;
  bool unit_norm = false, value_mix = false, first_values = false;
  float* slopes = nullptr;
  int rot_dims = 0;
  double rot_base = 0.0;
  float2* rotation = nullptr;        // [positions][rot_dims / 2]
  int64_t max_visible = 0;
  int mlp = TB_MLP_NONE;
  CacheGeom geom;
  void *k_cache = nullptr, *v_cache = nullptr;
  float *state1 = nullptr, *state2 = nullptr;
};

uint16_t* host_copy(std::vector<uint16_t>& buf, const uint16_t* src, size_t n, tb_space space) {
  buf.resize(n);
  if (space == TB_HOST) memcpy(buf.data(), src, n * 2);
  else if (cudaMemcpy(buf.data(), src, n * 2, cudaMemcpyDeviceToHost) != cudaSuccess) return nullptr;
  return buf.data();
}
float bf16_value(uint16_t b) {
  const uint32_t u = (uint32_t)b << 16;
  float f;
  memcpy(&f, &u, 4);
  return f;
}

}  // namespace

struct LayeredModel {
  tb_layered_config cfg;
  Precision prec = Precision::kBf16;
  int L = 0, B = 1, max_rows = 1, taps = 1, ring = 0;
  int width = 0, xs = 0;
  std::vector<LayerWeights> w;
  std::vector<LayerRun> runs;
  DenseWeight embed, head;         // head: without an image the embedding
  __nv_bfloat16* pos_table = nullptr;
  float *final_norm = nullptr, *embed_norm = nullptr;
  float* x[2] = {nullptr, nullptr};
  int32_t* pos = nullptr;
  float* rstd = nullptr;
  float* y = nullptr;              // partial sums of a product
  int64_t y_floats = 0;
  void *act_x = nullptr, *act_o = nullptr, *act_z = nullptr;
  void *act_c = nullptr, *act_q = nullptr, *act_v = nullptr;   // latent layers: query latent; per head the plain query, the attended latent
  void* act_l = nullptr;           // latents of a sequence as an operand, and what they are written out to: [positions][keys | values]
  __nv_bfloat16* expanded = nullptr;
  float *v_first = nullptr, *gates = nullptr;
  float2* part_ml = nullptr;       // splits of the flash attention, with flash_parts
  float* flash_parts = nullptr;
  int64_t flash_slots = 0;
  float* q = nullptr;
  __nv_bfloat16* q16 = nullptr;
  float *scores = nullptr, *part = nullptr;
  int64_t score_floats = 0;
  float* parts = nullptr;          // attention sums of CTAs that share a row's positions
  int64_t parts_rows = 0;
  float* snap = nullptr;
  int64_t rollback = 0;
  std::vector<void*> owned;        // every device allocation
};

namespace {

template <typename T>
tb_status dev_alloc(LayeredModel* m, T** p, size_t count, bool zero) {
  *p = nullptr;
  if (count == 0) return TB_OK;
  void* v = nullptr;
  const cudaError_t e = cudaMalloc(&v, count * sizeof(T));
  if (e != cudaSuccess)
    return fail(TB_ERR_OOM, "Out of memory allocating %zu MB on the device (%s)", count * sizeof(T) / (1024 * 1024), cudaGetErrorString(e));
  m->owned.push_back(v);
  if (zero) TB_CUDA_TRY(cudaMemset(v, 0, count * sizeof(T)));
  *p = static_cast<T*>(v);
  return TB_OK;
}

// A bf16 vector (plus `offset`) as fp32, zero-padded to `padded` elements.
tb_status dev_vector(LayeredModel* m, float** p, const uint16_t* src, int64_t n, int64_t padded, tb_space space, const char* what, float offset = 0.f) {
  if (!src) return fail(TB_ERR_ARG, "layered decoder: %s is missing", what);
  std::vector<uint16_t> h;
  if (!host_copy(h, src, (size_t)n, space)) return fail(TB_ERR_CUDA, "layered decoder: reading %s failed", what);
  std::vector<float> f((size_t)padded, 0.f);
  for (int64_t i = 0; i < n; ++i) f[(size_t)i] = offset + bf16_value(h[(size_t)i]);
  TB_TRY(dev_alloc(m, p, (size_t)padded, false));
  TB_CUDA_TRY(cudaMemcpy(*p, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice));
  return TB_OK;
}

// [width, taps] -> [taps][xs]
tb_status dev_taps(LayeredModel* m, float** p, const uint16_t* src, tb_space space) {
  *p = nullptr;
  if (!src) return TB_OK;
  std::vector<uint16_t> h;
  const int64_t n = m->width, t = m->taps;
  if (!host_copy(h, src, (size_t)(n * t), space)) return fail(TB_ERR_CUDA, "layered decoder: reading convolution weights failed");
  std::vector<float> f((size_t)(t * m->xs), 0.f);
  for (int64_t i = 0; i < n; ++i)
    for (int64_t j = 0; j < t; ++j) f[(size_t)(j * m->xs + i)] = bf16_value(h[(size_t)(i * t + j)]);
  TB_TRY(dev_alloc(m, p, f.size(), false));
  TB_CUDA_TRY(cudaMemcpy(*p, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice));
  return TB_OK;
}

tb_status dense_matrix(LayeredModel* m, DenseWeight* w, int64_t rows, int64_t k, int batch = 1) {
  TB_TRY(dense_weight_alloc(w, rows, k, batch));
  m->owned.push_back(w->img);
  return TB_OK;
}

// [q | k | v | gates] of a layer of heads, and their norms, biases and mixing.
tb_status load_heads(LayeredModel* m, LayerWeights& w, const tb_layered_layer& s, tb_space space) {
  w.kv_heads = s.num_kv_heads;
  w.dpad = (int)pad_to(w.dim, 16); w.vpad = (int)pad_to(w.vdim, 16);
  const int64_t nq = (int64_t)w.heads * w.dim, nk = (int64_t)w.kv_heads * w.dim, nv = (int64_t)w.kv_heads * w.vdim;
  w.q_off = 0;
  w.k_off = (int)pad_to(nq, 16);
  w.v_off = w.k_off + (int)pad_to(nk, 16);
  w.g_off = w.v_off + (int)pad_to(nv, 16);
  w.gate = s.gate_w != nullptr;
  w.qkv_cols = w.gate ? w.g_off + w.heads : w.v_off + nv;
  TB_TRY(dense_matrix(m, &w.qkv, w.qkv_cols, m->width));
  TB_TRY(dense_weight_fill(&w.qkv, w.q_off, s.q_w, nq, m->width, space));
  TB_TRY(dense_weight_fill(&w.qkv, w.k_off, s.k_w, nk, m->width, space));
  TB_TRY(dense_weight_fill(&w.qkv, w.v_off, s.v_w, nv, m->width, space));
  if (w.gate) TB_TRY(dense_weight_fill(&w.qkv, w.g_off, s.gate_w, w.heads, m->width, space));
  if (s.q_b || s.k_b || s.v_b) {
    std::vector<float> b((size_t)w.qkv.rows, 0.f);
    const struct { const uint16_t* src; int64_t n; int off; } seg[3] = {{s.q_b, nq, w.q_off}, {s.k_b, nk, w.k_off}, {s.v_b, nv, w.v_off}};
    for (const auto& g : seg) {
      if (!g.src) continue;
      std::vector<uint16_t> h;
      if (!host_copy(h, g.src, (size_t)g.n, space)) return fail(TB_ERR_CUDA, "layered decoder: reading a bias failed");
      for (int64_t j = 0; j < g.n; ++j) b[(size_t)(g.off + j)] = bf16_value(h[(size_t)j]);
    }
    TB_TRY(dev_alloc(m, &w.qkv_b, b.size(), false));
    TB_CUDA_TRY(cudaMemcpy(w.qkv_b, b.data(), b.size() * sizeof(float), cudaMemcpyHostToDevice));
  }
  if (s.q_norm) TB_TRY(dev_vector(m, &w.q_norm, s.q_norm, nq, nq, space, "q_norm"));
  if (s.k_norm) TB_TRY(dev_vector(m, &w.k_norm, s.k_norm, nk, nk, space, "k_norm"));
  if (s.talk) TB_TRY(dev_vector(m, &w.talk, s.talk, (int64_t)w.heads * w.heads, (int64_t)w.heads * w.heads, space, "talk"));
  if (s.vmix) {
    std::vector<uint16_t> h;
    if (!host_copy(h, s.vmix, 1, space)) return fail(TB_ERR_CUDA, "layered decoder: reading vmix failed");
    w.vmix = bf16_value(h[0]);
  }
  return TB_OK;
}

tb_status load_latent(LayeredModel* m, LayerWeights& w, const tb_layered_layer& s, tb_space space) {
  w.latent = true;
  w.kv_heads = 1;
  w.q_rank = s.q_rank; w.kv_rank = s.kv_rank; w.rot_dim = s.rot_dim;
  w.dpad = (int)pad_to(w.kv_rank + w.rot_dim, 16); w.vpad = (int)pad_to(w.kv_rank, 16);
  w.k_off = (int)pad_to(w.q_rank, 16);
  w.qkv_cols = w.k_off + w.kv_rank + w.rot_dim;
  TB_TRY(dense_matrix(m, &w.qkv, w.qkv_cols, m->width));
  TB_TRY(dense_weight_fill(&w.qkv, 0, s.dq_w, w.q_rank, m->width, space));
  TB_TRY(dense_weight_fill(&w.qkv, w.k_off, s.dkv_w, w.kv_rank + w.rot_dim, m->width, space));
  TB_TRY(dense_matrix(m, &w.uq, (int64_t)w.heads * (w.dim + w.rot_dim), w.q_rank));
  TB_TRY(dense_weight_fill(&w.uq, 0, s.uq_w, (int64_t)w.heads * (w.dim + w.rot_dim), w.q_rank, space));
  TB_TRY(dense_matrix(m, &w.uk, w.kv_rank, w.dim, w.heads));
  TB_TRY(dense_weight_fill(&w.uk, 0, s.uk_w, w.kv_rank, w.dim, space, true));
  TB_TRY(dense_matrix(m, &w.uv, w.vdim, w.kv_rank, w.heads));
  TB_TRY(dense_weight_fill(&w.uv, 0, s.uv_w, w.vdim, w.kv_rank, space));
  w.xpad = (int)pad_to(w.dim + w.rot_dim, 16);
  const int64_t row = (int64_t)w.heads * (w.dim + w.vdim);
  if (m->prec == Precision::kBf16 && flash_tc5_fits(w.xpad, w.vdim) && w.dim % 8 == 0 && w.rot_dim % 8 == 0 && w.kv_rank % 8 == 0 &&
      (size_t)(m->cfg.max_seq_len * row) * 2 <= kExpandBudget) {
    TB_TRY(dense_matrix(m, &w.ukv, row, w.kv_rank));
    TB_TRY(dense_weight_fill(&w.ukv, 0, s.uk_w, (int64_t)w.heads * w.dim, w.kv_rank, space));
    TB_TRY(dense_weight_fill(&w.ukv, (int64_t)w.heads * w.dim, s.uv_w, (int64_t)w.heads * w.vdim, w.kv_rank, space));
  }
  TB_TRY(dev_vector(m, &w.dq_norm, s.dq_norm, w.q_rank, w.q_rank, space, "dq_norm"));
  TB_TRY(dev_vector(m, &w.dkv_norm, s.dkv_norm, w.kv_rank, w.kv_rank, space, "dkv_norm"));
  return TB_OK;
}

tb_status load_weights(LayeredModel* m, int i, const tb_layered_layer& s, tb_space space) {
  LayerWeights& w = m->w[(size_t)i];
  w.heads = s.num_heads; w.dim = s.head_dim; w.vdim = s.value_dim;
  const float off = m->cfg.norm_offset;
  const int64_t no = (int64_t)w.heads * w.vdim;
  TB_TRY(s.mixer == TB_MIXER_LATENT ? load_latent(m, w, s, space) : load_heads(m, w, s, space));
  TB_TRY(dense_matrix(m, &w.o, m->width, no));
  TB_TRY(dense_weight_fill(&w.o, 0, s.o_w, m->width, no, space));
  if (s.o_b) TB_TRY(dev_vector(m, &w.o_b, s.o_b, m->width, m->xs, space, "o_b"));
  TB_TRY(dev_vector(m, &w.norm1, s.norm1, m->width, m->xs, space, "norm1", off));
  if (s.norm1_after) TB_TRY(dev_vector(m, &w.norm1b, s.norm1_after, m->width, m->xs, space, "norm1_after"));
  TB_TRY(dev_taps(m, &w.conv1, s.conv1, space));
  if (s.mlp != TB_MLP_NONE) {
    w.ff = s.ff;
    TB_TRY(dense_matrix(m, &w.up, w.ff, m->width));
    TB_TRY(dense_weight_fill(&w.up, 0, s.up_w, w.ff, m->width, space));
    TB_TRY(dense_matrix(m, &w.down, m->width, w.ff));
    TB_TRY(dense_weight_fill(&w.down, 0, s.down_w, m->width, w.ff, space));
    if (s.mlp == TB_MLP_POLYNORM) {
      if (!s.act) return fail(TB_ERR_ARG, "layered decoder: activation coefficients are missing (layer %d)", i);
      std::vector<uint16_t> h;
      if (!host_copy(h, s.act, 4, space)) return fail(TB_ERR_CUDA, "layered decoder: reading activation coefficients failed");
      for (int j = 0; j < 4; ++j) w.act[j] = bf16_value(h[(size_t)j]);
    }
    TB_TRY(dev_vector(m, &w.norm2, s.norm2, m->width, m->xs, space, "norm2", off));
    if (s.norm2_after) TB_TRY(dev_vector(m, &w.norm2b, s.norm2_after, m->width, m->xs, space, "norm2_after"));
    TB_TRY(dev_taps(m, &w.conv2, s.conv2, space));
  }
  return TB_OK;
}

// slope_h = 2^(-bias (h + 1) / heads)
tb_status dev_slopes(LayeredModel* m, float** p, int heads, double bias) {
  std::vector<float> f((size_t)heads);
  for (int h = 0; h < heads; ++h) f[(size_t)h] = (float)exp2(-bias * (h + 1) / heads);
  TB_TRY(dev_alloc(m, p, f.size(), false));
  TB_CUDA_TRY(cudaMemcpy(*p, f.data(), f.size() * sizeof(float), cudaMemcpyHostToDevice));
  return TB_OK;
}

tb_status create_impl(LayeredModel* m, const tb_layered_layer* layers, const LayeredTables& t, tb_space space, bool snapshots) {
  const tb_layered_config& c = m->cfg;
  const int64_t S = c.max_seq_len;
  const size_t esz = m->prec == Precision::kBf16 ? 2 : 4;
  TB_TRY(dense_matrix(m, &m->embed, c.vocab_size, m->width));
  TB_TRY(dense_weight_fill(&m->embed, 0, t.embed, c.vocab_size, m->width, space));
  if (t.head) {
    TB_TRY(dense_matrix(m, &m->head, c.vocab_size, m->width));
    TB_TRY(dense_weight_fill(&m->head, 0, t.head, c.vocab_size, m->width, space));
  }
  if (t.embed_norm) TB_TRY(dev_vector(m, &m->embed_norm, t.embed_norm, m->width, m->xs, space, "embed_norm", c.norm_offset));
  if (t.pos_table) {
    TB_TRY(dev_alloc(m, &m->pos_table, (size_t)(S * m->width), false));
    TB_CUDA_TRY(cudaMemcpy(m->pos_table, t.pos_table, (size_t)(S * m->width) * 2, space == TB_HOST ? cudaMemcpyHostToDevice : cudaMemcpyDeviceToDevice));
  }
  TB_TRY(dev_vector(m, &m->final_norm, t.final_norm, m->width, m->xs, space, "final_norm", c.norm_offset));
  m->w.resize((size_t)m->L);
  m->runs.resize((size_t)m->L);
  int64_t max_cols = m->embed.rows > 0 ? pad_to(m->width, 128) : 0, max_q = 0, max_o = 0, max_z = 0, max_score_row = 0, max_heads = 1;
  int64_t max_c = 0, max_qn = 0, max_ctx = 0, max_gates = 0, flash_vdim = 0, max_lat = 0, max_expanded = 0;
  const LayerRun* first_values = nullptr;
  m->rollback = m->ring - 2 * (m->taps - 1);
  for (int i = 0; i < m->L; ++i)
    if (layers[i].weights_of < 0) TB_TRY(load_weights(m, i, layers[i], space));
  for (int i = 0; i < m->L; ++i) {
    const tb_layered_layer& s = layers[i];
    LayerRun& r = m->runs[(size_t)i];
    int src = i;
    for (int hops = 0; layers[src].weights_of >= 0; ++hops) {
      if (layers[src].weights_of >= m->L || hops > m->L) return fail(TB_ERR_ARG, "layered decoder: weights_of of layer %d leads nowhere", i);
      src = layers[src].weights_of;
    }
    r.weights = src;
    const LayerWeights& w = m->w[(size_t)src];
    if ((s.mixer == TB_MIXER_LATENT) != w.latent || s.num_heads != w.heads || s.num_kv_heads != w.kv_heads || s.head_dim != w.dim || s.value_dim != w.vdim ||
        (w.latent && (s.q_rank != w.q_rank || s.kv_rank != w.kv_rank || s.rot_dim != w.rot_dim)) ||
        (s.mlp != TB_MLP_NONE) != (w.ff > 0) || (w.ff > 0 && s.ff != w.ff))
      return fail(TB_ERR_ARG, "layered decoder: layer %d and the layer whose weights it uses differ in size", i);
    r.scale = s.score_scale;
    r.mlp = s.mlp;
    r.softcap = s.score_softcap;
    r.unit_norm = s.qk_unit_norm != 0;
    r.value_mix = s.value_mix != 0;
    if (w.talk && (r.unit_norm || r.value_mix || w.gate || r.softcap != 0.f || s.distance_bias != 0.f || s.mask_chunk > 0))
      return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: mixed heads together with a score transform, chunks, value mixing or gates (layer %d)", i);
    if ((r.unit_norm || r.value_mix || w.gate) && (w.qkv_b || w.q_norm || w.k_norm))
      return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: per-head norms, value mixing or gates together with biases or norms of the whole projection (layer %d)", i);
    if (r.value_mix) {
      r.first_values = first_values == nullptr;
      if (first_values == nullptr) first_values = &r;
      const LayerWeights& f = m->w[(size_t)first_values->weights];
      if (w.kv_heads != f.kv_heads || w.vdim != f.vdim)
        return fail(TB_ERR_ARG, "layered decoder: the values of layer %d and those it mixes in differ in size", i);
    }
    if (s.distance_bias != 0.f) TB_TRY(dev_slopes(m, &r.slopes, w.heads, (double)s.distance_bias));
    r.rot_dims = w.latent ? s.rot_dims : 0;
    r.rot_base = s.rot_base;
    if (r.rot_dims > 0) {
      for (int j = 0; j < i && !r.rotation; ++j)
        if (m->runs[(size_t)j].rot_dims == r.rot_dims && m->runs[(size_t)j].rot_base == r.rot_base) r.rotation = m->runs[(size_t)j].rotation;
      if (!r.rotation) {
        TB_TRY(dev_alloc(m, &r.rotation, (size_t)(S * (r.rot_dims / 2)), false));
        TB_TRY(fill_rotation_table(r.rotation, S, r.rot_dims, r.rot_base));
      }
    }
    r.window = s.mask_window > 0 && s.mask_window < S ? s.mask_window : (int)S;
    r.keep_first = s.mask_keep_first < S ? s.mask_keep_first : (int)S;
    r.chunk = s.mask_chunk > 0 && s.mask_chunk < S ? s.mask_chunk : 0;
    const int reach = r.chunk > 0 && r.chunk < r.window ? r.chunk : r.window;   // the furthest key back is less than this away
    r.max_visible = (int64_t)reach + r.keep_first < S ? (int64_t)reach + r.keep_first : S;
    // ring behind the window or the chunk: everything the first row of a step sees must survive the rows appended with
    // it, and a sequence taken back by up to kHistory positions still finds its window
    const int64_t ring = pad_to((int64_t)reach + (m->max_rows > kHistory ? m->max_rows : kHistory), r.keep_first == 0 ? 128 : 1);   // 128: whole tiles of keys
    if (r.keep_first + ring < S) {
      r.geom.keep = r.keep_first;
      r.geom.ring = (int)ring;
      r.geom.rows = r.keep_first + ring;
      if (ring - reach + 1 < m->rollback) m->rollback = ring - reach + 1;
    } else {
      r.geom.rows = S;
    }
    char* kc = nullptr;
    TB_TRY(dev_alloc(m, &kc, (size_t)m->B * r.geom.rows * w.kv_heads * w.dpad * esz, true));
    r.k_cache = kc;
    if (!w.latent) {
      TB_TRY(dev_alloc(m, &kc, (size_t)m->B * r.geom.rows * w.kv_heads * w.vpad * esz, true));
      r.v_cache = kc;
    }
    if (w.conv1) TB_TRY(dev_alloc(m, &r.state1, (size_t)m->B * m->ring * m->xs, true));
    if (w.conv2) TB_TRY(dev_alloc(m, &r.state2, (size_t)m->B * m->ring * m->xs, true));
    if (w.qkv.rows > max_cols) max_cols = w.qkv.rows;
    if (w.up.rows > max_cols) max_cols = w.up.rows;
    if (w.uq.rows > max_cols) max_cols = w.uq.rows;
    auto most = [](int64_t& a, int64_t b) { if (b > a) a = b; };
    most(max_c, w.uq.kp);
    most(max_qn, w.heads * w.uk.kp);
    most(max_ctx, w.heads * w.uv.kp);
    if (w.gate) most(max_gates, w.heads);
    if (!w.talk) most(flash_vdim, w.latent && w.kv_rank > w.vdim ? w.kv_rank : w.vdim);
    if (w.ukv.img) {
      most(max_lat, w.ukv.kp);
      most(max_expanded, (int64_t)w.heads * (w.dim + w.vdim));
    }
    const int64_t q = (int64_t)w.heads * (w.dpad > w.xpad ? w.dpad : w.xpad);
    if (q > max_q) max_q = q;
    if (w.o.kp > max_o) max_o = w.o.kp;
    if (w.down.kp > max_z) max_z = w.down.kp;
    if (w.talk) most(max_score_row, (int64_t)w.heads * (int64_t)window_attn_score_stride(r.max_visible));
    if (w.heads > max_heads) max_heads = w.heads;
  }
  const int R = m->max_rows;
  const size_t rp = (size_t)dense_row_pad(R);
  for (auto& x : m->x) TB_TRY(dev_alloc(m, &x, (size_t)R * m->xs, true));
  TB_TRY(dev_alloc(m, &m->pos, (size_t)R, true));
  TB_TRY(dev_alloc(m, &m->rstd, (size_t)R, true));
  const int64_t y_rows = R > kMaxSplits * 64 ? R : kMaxSplits * 64;
  m->y_floats = y_rows * max_cols;
  TB_TRY(dev_alloc(m, &m->y, (size_t)m->y_floats, true));
  char* b = nullptr;
  TB_TRY(dev_alloc(m, &b, rp * m->xs * esz, true));
  m->act_x = b;
  TB_TRY(dev_alloc(m, &b, rp * max_o * esz, true));
  m->act_o = b;
  TB_TRY(dev_alloc(m, &b, rp * max_z * esz, true));
  m->act_z = b;
  TB_TRY(dev_alloc(m, &b, rp * max_c * esz, true));
  m->act_c = b;
  TB_TRY(dev_alloc(m, &b, rp * max_qn * esz, true));
  m->act_q = b;
  TB_TRY(dev_alloc(m, &b, rp * max_ctx * esz, true));
  m->act_v = b;
  if (max_lat > 0) {
    TB_TRY(dev_alloc(m, &b, (size_t)(dense_row_pad((int)S) * max_lat * 2), true));
    m->act_l = b;
    TB_TRY(dev_alloc(m, &m->expanded, (size_t)(S * max_expanded), true));
  }
  if (first_values) {
    const LayerWeights& f = m->w[(size_t)first_values->weights];
    TB_TRY(dev_alloc(m, &m->v_first, (size_t)R * f.kv_heads * f.vdim, true));
  }
  TB_TRY(dev_alloc(m, &m->gates, (size_t)(R * max_gates), true));
  TB_TRY(dev_alloc(m, &m->q, (size_t)(R * max_q), true));
  if (m->prec == Precision::kBf16) TB_TRY(dev_alloc(m, &m->q16, (size_t)(rp * max_q), true));
  if (max_score_row > 0) {   // layers with mixed heads
    int64_t srows = (int64_t)(kScoreBudget / 4) / max_score_row;
    if (srows < 1) srows = 1;
    if (srows > R) srows = R;
    m->score_floats = srows * max_score_row;
    TB_TRY(dev_alloc(m, &m->scores, (size_t)m->score_floats, false));
    TB_TRY(dev_alloc(m, &m->part, (size_t)(R * max_heads * kScoreSplitsMax * 2), false));
    m->parts_rows = 4 * R > 4 * kScoreSplitsMax ? 4 * R : 4 * kScoreSplitsMax;
    TB_TRY(dev_alloc(m, &m->parts, (size_t)m->parts_rows * max_o, false));
  }
  if (flash_vdim > 0 && m->prec == Precision::kBf16) {
    m->flash_slots = flash_part_slots(R, max_heads);
    TB_TRY(dev_alloc(m, &m->flash_parts, (size_t)(m->flash_slots * flash_vdim), false));
    TB_TRY(dev_alloc(m, &m->part_ml, (size_t)m->flash_slots, false));
  }
  if (snapshots) TB_TRY(dev_alloc(m, &m->snap, (size_t)m->L * R * m->xs, true));
  TB_CUDA_TRY(cudaDeviceSynchronize());
  return TB_OK;
}

}  // namespace

tb_status layered_create(LayeredModel** out, const tb_layered_config& c, const tb_layered_layer* layers, const LayeredTables& tables,
                         tb_space space, bool snapshots) {
  *out = nullptr;
  if (c.vocab_size <= 0 || c.hidden_size <= 0 || c.num_layers <= 0 || c.max_seq_len <= 0 || c.max_seq_len > (1 << 28))
    return fail(TB_ERR_ARG, "layered decoder: non-positive dimension");
  if (c.precision != TB_PRECISION_BF16 && c.precision != TB_PRECISION_F32) return fail(TB_ERR_ARG, "layered decoder: unknown precision %d", c.precision);
  if (c.conv_taps < 0 || c.conv_taps > 32) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: convolution over %d positions (at most 32)", c.conv_taps);
  for (int i = 0; i < c.num_layers; ++i) {
    const tb_layered_layer& s = layers[i];
    if (s.mixer != TB_MIXER_ATTENTION && s.mixer != TB_MIXER_LATENT) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: mixer kind %d (layer %d)", s.mixer, i);
    if (s.mlp != TB_MLP_NONE && s.mlp != TB_MLP_POLYNORM && s.mlp != TB_MLP_RELU2) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: feed-forward kind %d (layer %d)", s.mlp, i);
    if (s.num_heads <= 0 || s.num_kv_heads <= 0 || s.num_heads % s.num_kv_heads)
      return fail(TB_ERR_ARG, "num_heads (%d) must be divisible by num_kv_heads (%d) (layer %d)", s.num_heads, s.num_kv_heads, i);
    if (s.head_dim <= 0 || s.value_dim <= 0 || (s.mlp != TB_MLP_NONE && s.ff <= 0) || s.mask_keep_first < 0)
      return fail(TB_ERR_ARG, "layered decoder: non-positive size (layer %d)", i);
    if (s.mask_chunk < 0 || s.score_softcap < 0.f) return fail(TB_ERR_ARG, "layered decoder: negative chunk or cap (layer %d)", i);
    if (s.mixer == TB_MIXER_LATENT) {
      if (s.num_kv_heads != 1) return fail(TB_ERR_ARG, "layered decoder: latent attention has one key/value head, not %d (layer %d)", s.num_kv_heads, i);
      if (s.q_rank <= 0 || s.kv_rank <= 0 || s.rot_dim < 0 || s.rot_dims < 0 || s.rot_dims > s.rot_dim || s.rot_dims % 2 || (s.rot_dims > 0 && !(s.rot_base > 0.0)))
        return fail(TB_ERR_ARG, "layered decoder: bad latent or rotation size (layer %d)", i);
    }
  }
  LayeredModel* m = new (std::nothrow) LayeredModel();
  if (!m) return fail(TB_ERR_OOM, "layered decoder: host allocation failed");
  m->cfg = c;
  m->prec = c.precision == TB_PRECISION_F32 ? Precision::kF32 : Precision::kBf16;
  m->L = c.num_layers;
  m->B = c.max_batch <= 0 ? 1 : c.max_batch;
  m->max_rows = c.prefill_rows > m->B ? c.prefill_rows : m->B;
  m->width = (int)c.hidden_size;
  m->xs = (int)pad_to(c.hidden_size, kPad);
  m->taps = c.conv_taps > 0 ? c.conv_taps : 1;
  m->ring = 1;
  while (m->ring < kHistory + 2 * m->taps) m->ring *= 2;
  const tb_status s = create_impl(m, layers, tables, space, snapshots);
  if (s != TB_OK) {
    layered_destroy(m);
    return s;
  }
  *out = m;
  return TB_OK;
}

void layered_destroy(LayeredModel* m) {
  if (!m) return;
  for (void* p : m->owned) cudaFree(p);
  delete m;
}

int layered_max_rows(const LayeredModel* m) { return m->max_rows; }
int64_t layered_rollback(const LayeredModel* m) { return m->rollback; }
const float* layered_snapshot(const LayeredModel* m, int layer, int64_t* stride) {
  *stride = m->xs;
  return m->snap && layer >= 0 && layer < m->L ? m->snap + (size_t)layer * m->max_rows * m->xs : nullptr;
}

tb_status layered_enqueue(LayeredModel* m, const LayeredStep& s, cudaStream_t st, int* launches) {
  const int rows = s.r.rows;
  if (rows < 1 || rows > m->max_rows) return fail(TB_ERR_ARG, "layered step: %d rows (at most %d)", rows, m->max_rows);
  StepRows r = s.r;
  r.pos = m->pos;
  const Precision prec = m->prec;
  const int mp = dense_row_pad(rows);
  int n = 0, cur = 0;
  const ActOperand ax{m->act_x, mp, m->xs};

  // partial sums that the shared buffer holds of a product
  auto split_room = [&](const DenseWeight& w) -> int {
    const int64_t cap = m->y_floats / ((int64_t)rows * w.rows);
    return cap < kMaxSplits ? (int)cap : kMaxSplits;
  };
  // one product: partial sums into the shared buffer
  auto product = [&](const DenseWeight& w, const ActOperand& x, PartialSums* y) -> tb_status {
    const int64_t per = (int64_t)rows * w.rows;
    DenseGemmArgs a;
    a.w = &w; a.x = x; a.rows = rows; a.out = m->y; a.ldo = w.rows; a.n_valid = w.rows;
    a.splits = dense_splits(prec, w.rows, w.kp, rows, split_room(w));
    a.split_stride = (size_t)per;
    a.pdl = s.pdl;
    y->y = m->y; y->splits = a.splits; y->split_stride = a.split_stride; y->ldy = a.ldo;
    ++n;
    return launch_dense_gemm(prec, a, st);
  };
  GlueArgs g;                      // the glue in front of the next sublayer; its source is filled as we go
  auto reset_glue = [&] {
    g = GlueArgs();
    g.r = r; g.width = m->width; g.xs = m->xs; g.eps = m->cfg.norm_eps; g.taps = m->taps; g.ring = m->ring; g.pdl = s.pdl;
    g.neighbours = s.one_sequence && rows > 1;
  };
  auto glue = [&](const float* pre_w, const float* conv, float* state) -> tb_status {
    g.pre_w = pre_w; g.conv_w = conv; g.conv_state = state;
    g.rstd = conv != nullptr && rows >= kManyRows && s.one_sequence ? m->rstd : nullptr;
    g.out = ax;
    g.x_out = m->x[cur ^ 1];
    // Rows of this step may not overwrite inputs that other rows of it still read from the ring.
    const int room = m->ring - m->taps + 1;
    const bool direct = conv != nullptr && (rows <= room || !s.one_sequence);
    g.write_state = direct;
    TB_TRY(launch_glue(prec, g, st));
    n += g.rstd ? 2 : 1;
    cur ^= 1;
    if (conv != nullptr && !direct) {   // a long portion: its last inputs, once every row has been done
      GlueArgs t = g;
      t.conv_w = nullptr; t.out.data = nullptr; t.write_state = true;
      t.row0 = rows - room;
      TB_TRY(launch_glue(prec, t, st));
      ++n;
    }
    reset_glue();
    g.x_in = m->x[cur];
    return TB_OK;
  };

  // ---- mixers: the normed rows in ax -> operand of the output product ----
  auto flash = [&](FlashArgs& fa, const LayerRun& run) -> tb_status {
    fa.r = r; fa.k_cache = run.k_cache; fa.v_cache = run.v_cache; fa.geom = run.geom; fa.cache_slots = m->B;
    fa.scale = run.scale; fa.softcap = run.softcap; fa.slopes = run.slopes;
    fa.window = run.window; fa.keep_first = run.keep_first; fa.chunk = run.chunk; fa.max_visible = run.max_visible;
    fa.parts = m->flash_parts; fa.part_ml = m->part_ml; fa.part_slots = m->flash_slots;
    fa.q = prec == Precision::kBf16 ? static_cast<const void*>(m->q16) : m->q;
    fa.one_sequence = s.one_sequence; fa.pdl = s.pdl;
    return launch_flash_attention(prec, fa, st, &n);
  };
  auto mix_talk = [&](const LayerRun& run, const LayerWeights& w, QkvPrepArgs& qa, const ActOperand& out) -> tb_status {
    WindowAttnArgs wa;
    wa.r = r; wa.k_cache = run.k_cache; wa.v_cache = run.v_cache; wa.geom = run.geom;
    wa.heads = w.heads; wa.kv_heads = w.kv_heads; wa.dim = w.dim; wa.vdim = w.vdim; wa.dpad = w.dpad; wa.vpad = w.vpad;
    wa.scale = run.scale; wa.window = run.window; wa.keep_first = run.keep_first; wa.talk = w.talk; wa.max_visible = run.max_visible;
    wa.scores = m->scores; wa.part = m->part; wa.parts = m->parts; wa.parts_rows = m->parts_rows;
    wa.scratch_rows = m->score_floats / ((int64_t)w.heads * (int64_t)window_attn_score_stride(run.max_visible));
    wa.out = out;
    wa.one_sequence = s.one_sequence; wa.pdl = s.pdl;
    wa.q = m->q; wa.q16 = m->q16;
    const bool mma = prec == Precision::kBf16 && window_mma_supported(wa);
    qa.q = mma ? nullptr : m->q;
    qa.q16 = mma ? m->q16 : nullptr;
    TB_TRY(launch_qkv_prep(prec, qa, st));
    ++n;
    return launch_window_attention(prec, wa, st, &n);
  };
  auto mix_heads = [&](const LayerRun& run, const LayerWeights& w, const ActOperand& out) -> tb_status {
    PartialSums y;
    TB_TRY(product(w.qkv, ax, &y));
    FlashArgs fa;
    fa.heads = w.heads; fa.kv_heads = w.kv_heads; fa.dim = w.dim; fa.vdim = w.vdim; fa.dpad = w.dpad; fa.vpad = w.vpad;
    fa.gate = w.gate ? m->gates : nullptr;
    fa.unit_norm = run.unit_norm;
    fa.out = out;
    if (run.unit_norm || run.value_mix || w.gate) {
      HeadsPrepArgs ha;
      ha.r = r; ha.y = y;
      ha.heads = w.heads; ha.kv_heads = w.kv_heads; ha.dim = w.dim; ha.vdim = w.vdim; ha.dpad = w.dpad; ha.vpad = w.vpad;
      ha.q_off = w.q_off; ha.k_off = w.k_off; ha.v_off = w.v_off; ha.g_off = w.g_off;
      ha.unit_norm = run.unit_norm; ha.eps = m->cfg.norm_eps;
      ha.v_first = run.value_mix ? m->v_first : nullptr; ha.keep_first_values = run.first_values; ha.mix = w.vmix;
      ha.gate = w.gate ? m->gates : nullptr;
      ha.q = prec == Precision::kBf16 ? static_cast<void*>(m->q16) : m->q;
      ha.k_cache = run.k_cache; ha.v_cache = run.v_cache; ha.geom = run.geom; ha.pdl = s.pdl;
      TB_TRY(launch_heads_prep(prec, ha, st));
      ++n;
      return flash(fa, run);
    }
    QkvPrepArgs qa;
    qa.r = r; qa.y = y; qa.bias = w.qkv_b; qa.q_norm = w.q_norm; qa.k_norm = w.k_norm;
    qa.heads = w.heads; qa.kv_heads = w.kv_heads; qa.dim = w.dim; qa.vdim = w.vdim; qa.dpad = w.dpad; qa.vpad = w.vpad;
    qa.q_off = w.q_off; qa.k_off = w.k_off; qa.v_off = w.v_off; qa.eps = m->cfg.norm_eps;
    qa.k_cache = run.k_cache; qa.v_cache = run.v_cache; qa.geom = run.geom; qa.pdl = s.pdl;
    if (w.talk) return mix_talk(run, w, qa, out);
    qa.q = prec == Precision::kBf16 ? nullptr : m->q;
    qa.q16 = prec == Precision::kBf16 ? m->q16 : nullptr;
    TB_TRY(launch_qkv_prep(prec, qa, st));
    ++n;
    return flash(fa, run);
  };
  // a product per head whose sums are final
  auto head_product = [&](const DenseWeight& w, const ActOperand& x, int64_t features, DenseGemmArgs& a) -> tb_status {
    a.w = &w; a.x = x; a.rows = rows; a.n_valid = features; a.pdl = s.pdl;
    ++n;
    return launch_dense_gemm(prec, a, st);
  };
  auto mix_latent = [&](const LayerRun& run, const LayerWeights& w, const ActOperand& out) -> tb_status {
    PartialSums y;
    TB_TRY(product(w.qkv, ax, &y));
    LatentPrepArgs la;
    la.r = r; la.y = y; la.q_rank = w.q_rank; la.kv_rank = w.kv_rank; la.rot_dim = w.rot_dim; la.rot_dims = run.rot_dims;
    la.kv_off = w.k_off; la.dpad = w.dpad; la.q_norm = w.dq_norm; la.kv_norm = w.dkv_norm; la.table = run.rotation; la.eps = m->cfg.norm_eps;
    la.out = ActOperand{m->act_c, mp, (int)w.uq.kp};
    la.cache = run.k_cache; la.geom = run.geom; la.pdl = s.pdl;
    TB_TRY(launch_latent_prep(prec, la, st));
    TB_TRY(product(w.uq, la.out, &y));
    LatentQueryArgs lq;
    lq.r = r; lq.y = y; lq.heads = w.heads; lq.dim = w.dim; lq.rot_dim = w.rot_dim; lq.rot_dims = run.rot_dims;
    lq.table = run.rotation; lq.pdl = s.pdl;
    lq.q = prec == Precision::kBf16 ? static_cast<void*>(m->q16) : m->q;
    if (w.ukv.img && s.one_sequence && s.start >= 0 && rows >= kExpandRows && run.keep_first == 0) {
      // a portion: fewer operations with the keys and values of what it sees written out for this layer
      lq.dpad = w.xpad; lq.rot_at = w.dim;
      TB_TRY(launch_latent_query(prec, lq, st));
      LatentRowsArgs lr;
      lr.r = r; lr.cache = run.k_cache; lr.geom = run.geom; lr.kv_rank = w.kv_rank; lr.dpad = w.dpad; lr.pdl = s.pdl;
      lr.lo = VisibleRange((int)s.start, run.window, 0, run.chunk).lo / 128 * 128;   // whole tiles of keys
      lr.n = (int)s.start + rows - lr.lo;
      lr.out = ActOperand{m->act_l, dense_row_pad(lr.n), (int)w.ukv.kp};
      TB_TRY(launch_latent_rows(lr, st));
      const int64_t row = (int64_t)w.heads * (w.dim + w.vdim);
      DenseGemmArgs xa;
      xa.w = &w.ukv; xa.x = lr.out; xa.rows = lr.n; xa.n_valid = row; xa.pdl = s.pdl;
      xa.sink = DenseSink::kRows; xa.out = m->expanded; xa.ldo = row;
      TB_TRY(launch_dense_gemm(prec, xa, st));
      n += 4;
      FlashArgs fa;
      fa.heads = fa.kv_heads = w.heads; fa.dim = w.dim + w.rot_dim; fa.vdim = w.vdim; fa.dpad = w.xpad; fa.vpad = (int)pad_to(w.vdim, 16);
      fa.key_rows = m->expanded; fa.value_rows = m->expanded + (int64_t)w.heads * w.dim;
      fa.key_cols = w.dim; fa.key_base = lr.lo; fa.key_count = lr.n; fa.row_stride = (int)row; fa.rest_col = w.kv_rank; fa.cache_row = w.dpad;
      fa.out = out;
      return flash(fa, run);
    }
    lq.dpad = w.dpad; lq.rot_at = w.kv_rank;
    lq.out = ActOperand{m->act_q, mp, (int)w.uk.kp};
    TB_TRY(launch_latent_query(prec, lq, st));
    n += 2;
    DenseGemmArgs ka;
    ka.sink = DenseSink::kRows; ka.out = lq.q; ka.ldo = (int64_t)w.heads * w.dpad; ka.batch_cols = w.dpad;
    TB_TRY(head_product(w.uk, lq.out, w.kv_rank, ka));
    FlashArgs fa;
    fa.heads = w.heads; fa.kv_heads = 1; fa.dim = w.kv_rank + w.rot_dim; fa.vdim = w.kv_rank; fa.dpad = w.dpad; fa.vpad = w.vpad;
    fa.values_in_keys = true; fa.out_per_head = true;
    fa.out = ActOperand{m->act_v, mp, (int)w.uv.kp};
    TB_TRY(flash(fa, run));
    DenseGemmArgs va;
    va.sink = DenseSink::kOperand; va.operand = out; va.batch_cols = w.vdim;
    return head_product(w.uv, fa.out, w.vdim, va);
  };
  // up product and activation -> operand of the down product
  auto feed_forward = [&](const LayerRun& run, const LayerWeights& w, const ActOperand& out) -> tb_status {
    PartialSums y;
    if (run.mlp == TB_MLP_RELU2) {
      double gain = 0.0;
      dense_splits(prec, w.up.rows, w.up.kp, rows, split_room(w.up), &gain);
      if (gain < kLaunchStages) {   // the activation in the product's epilogue
        DenseGemmArgs a;
        a.w = &w.up; a.x = ax; a.rows = rows; a.n_valid = out.kp; a.pdl = s.pdl;
        a.sink = DenseSink::kOperand; a.operand = out; a.act = DenseAct::kRelu2;
        ++n;
        return launch_dense_gemm(prec, a, st);
      }
      TB_TRY(product(w.up, ax, &y));
      ++n;
      return launch_relu2(prec, rows, y, out, s.pdl, st);
    }
    TB_TRY(product(w.up, ax, &y));
    PolyNormArgs pa;
    pa.rows = rows; pa.z = y; pa.width = (int)w.ff; pa.eps = m->cfg.norm_eps; pa.pdl = s.pdl;
    for (int j = 0; j < 4; ++j) pa.coef[j] = w.act[j];
    pa.out = out;
    ++n;
    return launch_poly_norm(prec, pa, st);
  };

  reset_glue();
  g.post_w = m->embed_norm;
  g.embed = m->embed; g.embed_scale = m->cfg.embed_scale; g.pos_table = m->pos_table; g.vocab = m->cfg.vocab_size; g.max_pos = m->cfg.max_seq_len;
  for (int l = 0; l < m->L; ++l) {
    const LayerRun& run = m->runs[(size_t)l];
    const LayerWeights& w = m->w[(size_t)run.weights];
    TB_TRY(glue(w.norm1, w.conv1, run.state1));
    const ActOperand ao{m->act_o, mp, (int)w.o.kp}, az{m->act_z, mp, (int)w.down.kp};
    TB_TRY(w.latent ? mix_latent(run, w, ao) : mix_heads(run, w, ao));
    PartialSums y;
    TB_TRY(product(w.o, ao, &y));
    g.y = y; g.y_bias = w.o_b; g.post_w = w.norm1b;
    if (run.mlp != TB_MLP_NONE) {
      TB_TRY(glue(w.norm2, w.conv2, run.state2));
      TB_TRY(feed_forward(run, w, az));
      TB_TRY(product(w.down, az, &y));
      g.y = y; g.y_bias = nullptr; g.post_w = w.norm2b;
    }
    if (s.snapshots && m->snap) g.snapshot = m->snap + (size_t)l * m->max_rows * m->xs;
  }
  if (s.before_lm_head) TB_CUDA_TRY(cudaEventRecord(s.before_lm_head, st));
  if (s.logit_rows > 0 || g.snapshot) {
    // the final norm, for the rows whose logits are wanted, and the output matrix
    const ActOperand af{m->act_x, dense_row_pad(s.logit_rows > 0 ? s.logit_rows : 1), m->xs};
    g.pre_w = m->final_norm;
    g.x_out = m->x[cur ^ 1];
    if (s.logit_rows > 0) g.out = af;
    g.row_map = s.row_map;
    TB_TRY(launch_glue(prec, g, st));
    n += g.rstd ? 2 : 1;
    if (s.logit_rows > 0) {
      DenseGemmArgs a;
      a.w = m->head.img ? &m->head : &m->embed; a.x = af; a.rows = s.logit_rows; a.out = s.logits; a.ldo = m->cfg.vocab_size; a.n_valid = m->cfg.vocab_size;
      a.pdl = s.pdl;
      TB_TRY(launch_dense_gemm(prec, a, st));
      ++n;
    }
  }
  *launches = n;
  return TB_OK;
}

}  // namespace tb

// The layered decoder: a stack of sublayers (mixer, optional feed-forward), each
//   x <- x + [norm_after] f(h + conv(h)),  h = norm_before(x)
// with its constants and sizes taken per layer from the caller.  Layers may share weights (weights_of); each
// run of a layer has its own cache and convolution states.
//
// One step is a chain of kernels per layer
//   glue (residual, norms, convolution) -> QKV product -> query/key norm + cache append -> scores -> mix ->
//   output product -> glue -> up product -> PolyNorm -> down product
// and the final norm with the tied output product for the rows whose logits are wanted.  Every buffer between
// two kernels is written by exactly one of them and read by the next, so one buffer of partial sums and one
// operand buffer per kind serve the whole stack; the residual stream alternates between two buffers because
// the convolution recomputes its neighbours' rows.
//
// State of a sequence: per layer the rows of K and V (a ring behind a window: window + a portion's rows +
// room to go back; the kept first positions have rows of their own) and per sublayer the last inputs of the
// convolution, by position in a ring.
#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "layered.cuh"

namespace tb {

namespace {

constexpr int kHistory = 128;      // positions a sequence can always be taken back
constexpr int kMaxSplits = 8;
constexpr size_t kScoreBudget = 1024u << 20;
constexpr int kManyRows = 64;       // from here on the glue is two kernels

struct LayerWeights {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dpad = 0, vpad = 0;
  int q_off = 0, k_off = 0, v_off = 0;
  int64_t qkv_cols = 0;
  int64_t ff = 0;
  float act[4] = {0, 0, 0, 0};
  DenseWeight qkv, o, up, down;
  float *qkv_b = nullptr, *q_norm = nullptr, *k_norm = nullptr, *talk = nullptr, *o_b = nullptr;
  float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
  float *conv1 = nullptr, *conv2 = nullptr;
};

struct LayerRun {
  int weights = 0;                 // index of the layer that owns the weights
  float scale = 1.f;
  int window = 0, keep_first = 0;
  int64_t max_visible = 0;
  bool mlp = false;
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
  DenseWeight embed;
  __nv_bfloat16* pos_table = nullptr;
  float* final_norm = nullptr;
  float* x[2] = {nullptr, nullptr};
  int32_t* pos = nullptr;
  float* rstd = nullptr;
  float* y = nullptr;              // partial sums of a product
  int64_t y_floats = 0;
  void *act_x = nullptr, *act_o = nullptr, *act_z = nullptr;
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

// A bf16 vector as fp32, zero-padded to `padded` elements.
tb_status dev_vector(LayeredModel* m, float** p, const uint16_t* src, int64_t n, int64_t padded, tb_space space, const char* what) {
  if (!src) return fail(TB_ERR_ARG, "layered decoder: %s is missing", what);
  std::vector<uint16_t> h;
  if (!host_copy(h, src, (size_t)n, space)) return fail(TB_ERR_CUDA, "layered decoder: reading %s failed", what);
  std::vector<float> f((size_t)padded, 0.f);
  for (int64_t i = 0; i < n; ++i) f[(size_t)i] = bf16_value(h[(size_t)i]);
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

tb_status dense_matrix(LayeredModel* m, DenseWeight* w, int64_t rows, int64_t k) {
  TB_TRY(dense_weight_alloc(w, rows, k));
  m->owned.push_back(w->img);
  return TB_OK;
}

tb_status load_weights(LayeredModel* m, int i, const tb_layered_layer& s, tb_space space) {
  LayerWeights& w = m->w[(size_t)i];
  w.heads = s.num_heads; w.kv_heads = s.num_kv_heads; w.dim = s.head_dim; w.vdim = s.value_dim;
  w.dpad = (int)pad_to(w.dim, 16); w.vpad = (int)pad_to(w.vdim, 16);
  const int64_t nq = (int64_t)w.heads * w.dim, nk = (int64_t)w.kv_heads * w.dim, nv = (int64_t)w.kv_heads * w.vdim, no = (int64_t)w.heads * w.vdim;
  w.q_off = 0;
  w.k_off = (int)pad_to(nq, 16);
  w.v_off = w.k_off + (int)pad_to(nk, 16);
  w.qkv_cols = w.v_off + nv;
  TB_TRY(dense_matrix(m, &w.qkv, w.qkv_cols, m->width));
  TB_TRY(dense_weight_fill(&w.qkv, w.q_off, s.q_w, nq, m->width, space));
  TB_TRY(dense_weight_fill(&w.qkv, w.k_off, s.k_w, nk, m->width, space));
  TB_TRY(dense_weight_fill(&w.qkv, w.v_off, s.v_w, nv, m->width, space));
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
  if (s.talk) {
    TB_TRY(dev_vector(m, &w.talk, s.talk, (int64_t)w.heads * w.heads, (int64_t)w.heads * w.heads, space, "talk"));
  } else {   // heads not mixed
    std::vector<float> id((size_t)w.heads * w.heads, 0.f);
    for (int h = 0; h < w.heads; ++h) id[(size_t)h * w.heads + h] = 1.f;
    TB_TRY(dev_alloc(m, &w.talk, id.size(), false));
    TB_CUDA_TRY(cudaMemcpy(w.talk, id.data(), id.size() * sizeof(float), cudaMemcpyHostToDevice));
  }
  TB_TRY(dense_matrix(m, &w.o, m->width, no));
  TB_TRY(dense_weight_fill(&w.o, 0, s.o_w, m->width, no, space));
  if (s.o_b) TB_TRY(dev_vector(m, &w.o_b, s.o_b, m->width, m->xs, space, "o_b"));
  TB_TRY(dev_vector(m, &w.norm1, s.norm1, m->width, m->xs, space, "norm1"));
  if (s.norm1_after) TB_TRY(dev_vector(m, &w.norm1b, s.norm1_after, m->width, m->xs, space, "norm1_after"));
  TB_TRY(dev_taps(m, &w.conv1, s.conv1, space));
  if (s.mlp != TB_MLP_NONE) {
    w.ff = s.ff;
    TB_TRY(dense_matrix(m, &w.up, w.ff, m->width));
    TB_TRY(dense_weight_fill(&w.up, 0, s.up_w, w.ff, m->width, space));
    TB_TRY(dense_matrix(m, &w.down, m->width, w.ff));
    TB_TRY(dense_weight_fill(&w.down, 0, s.down_w, m->width, w.ff, space));
    if (!s.act) return fail(TB_ERR_ARG, "layered decoder: activation coefficients are missing (layer %d)", i);
    std::vector<uint16_t> h;
    if (!host_copy(h, s.act, 4, space)) return fail(TB_ERR_CUDA, "layered decoder: reading activation coefficients failed");
    for (int j = 0; j < 4; ++j) w.act[j] = bf16_value(h[(size_t)j]);
    TB_TRY(dev_vector(m, &w.norm2, s.norm2, m->width, m->xs, space, "norm2"));
    if (s.norm2_after) TB_TRY(dev_vector(m, &w.norm2b, s.norm2_after, m->width, m->xs, space, "norm2_after"));
    TB_TRY(dev_taps(m, &w.conv2, s.conv2, space));
  }
  return TB_OK;
}

tb_status create_impl(LayeredModel* m, const tb_layered_layer* layers, const uint16_t* embed, const uint16_t* pos_table,
                      const uint16_t* final_norm, tb_space space, bool snapshots) {
  const tb_layered_config& c = m->cfg;
  const int64_t S = c.max_seq_len;
  const size_t esz = m->prec == Precision::kBf16 ? 2 : 4;
  TB_TRY(dense_matrix(m, &m->embed, c.vocab_size, m->width));
  TB_TRY(dense_weight_fill(&m->embed, 0, embed, c.vocab_size, m->width, space));
  if (pos_table) {
    TB_TRY(dev_alloc(m, &m->pos_table, (size_t)(S * m->width), false));
    TB_CUDA_TRY(cudaMemcpy(m->pos_table, pos_table, (size_t)(S * m->width) * 2, space == TB_HOST ? cudaMemcpyHostToDevice : cudaMemcpyDeviceToDevice));
  }
  TB_TRY(dev_vector(m, &m->final_norm, final_norm, m->width, m->xs, space, "final_norm"));
  m->w.resize((size_t)m->L);
  m->runs.resize((size_t)m->L);
  int64_t max_cols = m->embed.rows > 0 ? pad_to(m->width, 128) : 0, max_q = 0, max_o = 0, max_z = 0, max_score_row = 1, max_heads = 1;
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
    if (s.num_heads != w.heads || s.num_kv_heads != w.kv_heads || s.head_dim != w.dim || s.value_dim != w.vdim ||
        (s.mlp != TB_MLP_NONE) != (w.ff > 0) || (w.ff > 0 && s.ff != w.ff))
      return fail(TB_ERR_ARG, "layered decoder: layer %d and the layer whose weights it uses differ in size", i);
    r.scale = s.score_scale;
    r.mlp = s.mlp != TB_MLP_NONE;
    r.window = s.mask_window > 0 && s.mask_window < S ? s.mask_window : (int)S;
    r.keep_first = s.mask_keep_first < S ? s.mask_keep_first : (int)S;
    r.max_visible = (int64_t)r.window + r.keep_first < S ? (int64_t)r.window + r.keep_first : S;
    // ring behind the window: everything the first row of a step sees must survive the rows appended with
    // it, and a sequence taken back by up to kHistory positions still finds its window
    const int64_t ring = (int64_t)r.window + (m->max_rows > kHistory ? m->max_rows : kHistory);
    if (r.keep_first + ring < S) {
      r.geom.keep = r.keep_first;
      r.geom.ring = (int)ring;
      r.geom.rows = r.keep_first + ring;
      if (ring - r.window + 1 < m->rollback) m->rollback = ring - r.window + 1;
    } else {
      r.geom.rows = S;
    }
    char* kc = nullptr;
    TB_TRY(dev_alloc(m, &kc, (size_t)m->B * r.geom.rows * w.kv_heads * w.dpad * esz, true));
    r.k_cache = kc;
    TB_TRY(dev_alloc(m, &kc, (size_t)m->B * r.geom.rows * w.kv_heads * w.vpad * esz, true));
    r.v_cache = kc;
    if (w.conv1) TB_TRY(dev_alloc(m, &r.state1, (size_t)m->B * m->ring * m->xs, true));
    if (w.conv2) TB_TRY(dev_alloc(m, &r.state2, (size_t)m->B * m->ring * m->xs, true));
    if (w.qkv.rows > max_cols) max_cols = w.qkv.rows;
    if (w.up.rows > max_cols) max_cols = w.up.rows;
    const int64_t q = (int64_t)w.heads * w.dpad;
    if (q > max_q) max_q = q;
    if (w.o.kp > max_o) max_o = w.o.kp;
    if (w.down.kp > max_z) max_z = w.down.kp;
    const int64_t sr = (int64_t)w.heads * (int64_t)window_attn_score_stride(r.max_visible);
    if (sr > max_score_row) max_score_row = sr;
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
  TB_TRY(dev_alloc(m, &m->q, (size_t)(R * max_q), true));
  if (m->prec == Precision::kBf16) TB_TRY(dev_alloc(m, &m->q16, (size_t)(rp * max_q), true));
  int64_t srows = (int64_t)(kScoreBudget / 4) / max_score_row;
  if (srows < 1) srows = 1;
  if (srows > R) srows = R;
  
  m->score_floats = srows * max_score_row;
  TB_TRY(dev_alloc(m, &m->scores, (size_t)m->score_floats, false));
  TB_TRY(dev_alloc(m, &m->part, (size_t)(R * max_heads * kScoreSplitsMax * 2), false));
  m->parts_rows = 4 * R > 4 * kScoreSplitsMax ? 4 * R : 4 * kScoreSplitsMax;
  TB_TRY(dev_alloc(m, &m->parts, (size_t)m->parts_rows * max_o, false));
  if (snapshots) TB_TRY(dev_alloc(m, &m->snap, (size_t)m->L * R * m->xs, true));
  TB_CUDA_TRY(cudaDeviceSynchronize());
  return TB_OK;
}

}  // namespace

tb_status layered_create(LayeredModel** out, const tb_layered_config& c, const tb_layered_layer* layers, const uint16_t* embed,
                         const uint16_t* pos_table, const uint16_t* final_norm, tb_space space, bool snapshots) {
  *out = nullptr;
  if (c.vocab_size <= 0 || c.hidden_size <= 0 || c.num_layers <= 0 || c.max_seq_len <= 0 || c.max_seq_len > (1 << 28))
    return fail(TB_ERR_ARG, "layered decoder: non-positive dimension");
  if (c.precision != TB_PRECISION_BF16 && c.precision != TB_PRECISION_F32) return fail(TB_ERR_ARG, "layered decoder: unknown precision %d", c.precision);
  if (c.conv_taps < 0 || c.conv_taps > 32) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: convolution over %d positions (at most 32)", c.conv_taps);
  for (int i = 0; i < c.num_layers; ++i) {
    const tb_layered_layer& s = layers[i];
    if (s.mixer != TB_MIXER_ATTENTION) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: mixer kind %d (layer %d)", s.mixer, i);
    if (s.mlp != TB_MLP_NONE && s.mlp != TB_MLP_POLYNORM) return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: feed-forward kind %d (layer %d)", s.mlp, i);
    if (s.num_heads <= 0 || s.num_kv_heads <= 0 || s.num_heads % s.num_kv_heads)
      return fail(TB_ERR_ARG, "num_heads (%d) must be divisible by num_kv_heads (%d) (layer %d)", s.num_heads, s.num_kv_heads, i);
    if (s.head_dim <= 0 || s.value_dim <= 0 || (s.mlp != TB_MLP_NONE && s.ff <= 0) || s.mask_keep_first < 0)
      return fail(TB_ERR_ARG, "layered decoder: non-positive size (layer %d)", i);
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
  const tb_status s = create_impl(m, layers, embed, pos_table, final_norm, space, snapshots);
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

  // one product: partial sums into the shared buffer
  auto product = [&](const DenseWeight& w, const ActOperand& x, PartialSums* y) -> tb_status {
    const int64_t per = (int64_t)rows * w.rows;
    int64_t cap = m->y_floats / per;
    if (cap > kMaxSplits) cap = kMaxSplits;
    DenseGemmArgs a;
    a.w = &w; a.x = x; a.rows = rows; a.out = m->y; a.ldo = w.rows; a.n_valid = w.rows;
    a.splits = dense_splits(prec, w.rows, w.kp, rows, (int)cap);
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
    g.rstd = rows >= kManyRows && s.one_sequence ? m->rstd : nullptr;
    g.neighbours = s.one_sequence && rows > 1;
  };
  auto glue = [&](const float* pre_w, const float* conv, float* state) -> tb_status {
    g.pre_w = pre_w; g.conv_w = conv; g.conv_state = state;
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

  reset_glue();
  g.embed = m->embed; g.embed_scale = m->cfg.embed_scale; g.pos_table = m->pos_table; g.vocab = m->cfg.vocab_size; g.max_pos = m->cfg.max_seq_len;
  for (int l = 0; l < m->L; ++l) {
    const LayerRun& run = m->runs[(size_t)l];
    const LayerWeights& w = m->w[(size_t)run.weights];
    TB_TRY(glue(w.norm1, w.conv1, run.state1));
    PartialSums y;
    TB_TRY(product(w.qkv, ax, &y));
    QkvPrepArgs qa;
    qa.r = r; qa.y = y; qa.bias = w.qkv_b; qa.q_norm = w.q_norm; qa.k_norm = w.k_norm;
    qa.heads = w.heads; qa.kv_heads = w.kv_heads; qa.dim = w.dim; qa.vdim = w.vdim; qa.dpad = w.dpad; qa.vpad = w.vpad;
    qa.q_off = w.q_off; qa.k_off = w.k_off; qa.v_off = w.v_off; qa.eps = m->cfg.norm_eps;
    qa.k_cache = run.k_cache; qa.v_cache = run.v_cache; qa.geom = run.geom; qa.pdl = s.pdl;
    WindowAttnArgs wa;
    wa.r = r; wa.k_cache = run.k_cache; wa.v_cache = run.v_cache; wa.geom = run.geom;
    wa.heads = w.heads; wa.kv_heads = w.kv_heads; wa.dim = w.dim; wa.vdim = w.vdim; wa.dpad = w.dpad; wa.vpad = w.vpad;
    wa.scale = run.scale; wa.window = run.window; wa.keep_first = run.keep_first; wa.talk = w.talk; wa.max_visible = run.max_visible;
    wa.scores = m->scores; wa.part = m->part; wa.parts = m->parts; wa.parts_rows = m->parts_rows;
    wa.scratch_rows = m->score_floats / ((int64_t)w.heads * (int64_t)window_attn_score_stride(run.max_visible));
    wa.out = ActOperand{m->act_o, mp, (int)w.o.kp};
    wa.one_sequence = s.one_sequence; wa.pdl = s.pdl;
    wa.q = m->q; wa.q16 = m->q16;
    const bool mma = prec == Precision::kBf16 && window_mma_supported(wa);
    qa.q = mma ? nullptr : m->q;
    qa.q16 = mma ? m->q16 : nullptr;
    TB_TRY(launch_qkv_prep(prec, qa, st));
    ++n;
    TB_TRY(launch_window_attention(prec, wa, st, &n));
    TB_TRY(product(w.o, wa.out, &y));
    g.y = y; g.y_bias = w.o_b; g.post_w = w.norm1b;
    if (run.mlp) {
      TB_TRY(glue(w.norm2, w.conv2, run.state2));
      TB_TRY(product(w.up, ax, &y));
      PolyNormArgs pa;
      pa.rows = rows; pa.z = y; pa.width = (int)w.ff; pa.eps = m->cfg.norm_eps; pa.pdl = s.pdl;
      for (int j = 0; j < 4; ++j) pa.coef[j] = w.act[j];
      pa.out = ActOperand{m->act_z, mp, (int)w.down.kp};
      TB_TRY(launch_poly_norm(prec, pa, st));
      ++n;
      TB_TRY(product(w.down, pa.out, &y));
      g.y = y; g.y_bias = nullptr; g.post_w = w.norm2b;
    }
    if (s.snapshots && m->snap) g.snapshot = m->snap + (size_t)l * m->max_rows * m->xs;
  }
  if (s.before_lm_head) TB_CUDA_TRY(cudaEventRecord(s.before_lm_head, st));
  if (s.logit_rows > 0 || g.snapshot) {
    // the final norm, for the rows whose logits are wanted, and the tied output matrix
    const ActOperand af{m->act_x, dense_row_pad(s.logit_rows > 0 ? s.logit_rows : 1), m->xs};
    g.pre_w = m->final_norm;
    g.x_out = m->x[cur ^ 1];
    if (s.logit_rows > 0) g.out = af;
    g.row_map = s.row_map;
    TB_TRY(launch_glue(prec, g, st));
    n += g.rstd ? 2 : 1;
    if (s.logit_rows > 0) {
      DenseGemmArgs a;
      a.w = &m->embed; a.x = af; a.rows = s.logit_rows; a.out = s.logits; a.ldo = m->cfg.vocab_size; a.n_valid = m->cfg.vocab_size;
      a.pdl = s.pdl;
      TB_TRY(launch_dense_gemm(prec, a, st));
      ++n;
    }
  }
  *launches = n;
  return TB_OK;
}

}  // namespace tb

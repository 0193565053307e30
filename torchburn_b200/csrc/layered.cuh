// A decoder-only model described layer by layer (tb_layered_config / tb_layered_layer), behind the same
// tb_decoder handle as the INT4 models: device weights, caches and convolution states, and the enqueueing of
// one step.
#pragma once

#include "dense.cuh"

namespace tb {

struct LayeredModel;

struct LayeredStep {
  StepRows r;                      // tokens / slots / offsets on the device
  bool one_sequence = false;       // the rows are consecutive positions of one sequence
  int64_t start = -1;              // then the first row's position, where the host knows it
  const int32_t* row_map = nullptr;  // row -> logits row or -1; null: every row in place
  int logit_rows = 0;
  float* logits = nullptr;         // [logit_rows, vocab]
  bool pdl = false;
  bool snapshots = false;          // keep the residual stream after every layer
  cudaEvent_t before_lm_head = nullptr;
};

struct LayeredTables {
  const uint16_t* embed = nullptr;
  const uint16_t* embed_norm = nullptr;   // or null
  const uint16_t* pos_table = nullptr;    // or null
  const uint16_t* final_norm = nullptr;
  const uint16_t* head = nullptr;         // null: embed
};
tb_status layered_create(LayeredModel** out, const tb_layered_config& c, const tb_layered_layer* layers, const LayeredTables& tables,
                         tb_space space, bool snapshots);
void layered_destroy(LayeredModel* m);
int layered_max_rows(const LayeredModel* m);      // rows of one step
// How far back of the furthest position written a sequence may be continued (its rings hold that much).
int64_t layered_rollback(const LayeredModel* m);
tb_status layered_enqueue(LayeredModel* m, const LayeredStep& s, cudaStream_t st, int* launches);
// The residual stream after layer `layer` of the last step with snapshots: device rows with stride *stride.
const float* layered_snapshot(const LayeredModel* m, int layer, int64_t* stride);

}  // namespace tb

// Stands in for the INT4 kernels in a library built without them (build.py, profile "dense"): every launch
// fails with TB_ERR_UNSUPPORTED, the tuning hooks do nothing and no fault is ever reported.
#include "tb_common.cuh"

namespace tb {

namespace {
tb_status absent() { return fail(TB_ERR_UNSUPPORTED, "TB_UNSUPPORTED: this build of the library has no INT4 kernels (python -m torchburn_b200.build)"); }
}  // namespace

tb_status launch_w4_gemv(const GemvArgs&, cudaStream_t) { return absent(); }
int w4_gemv_launches(const GemvArgs&) { return 0; }
void release_workspaces() {}
void set_gemv_tuning(int, int, int) {}
size_t w4_mma_scratch_bytes(int, int64_t) { return 0; }
int tc5_fault_flag() { return 0; }
void set_stream_tuning(int, int, int, int, int) {}
int stream_fault_flag() { return 0; }
size_t attention_scratch_bytes(int, int, int, int, int64_t) { return 0; }
size_t attention_counters_offset(int, int, int, int, int64_t, size_t* n) {
  if (n) *n = 0;
  return 0;
}
void set_attention_chunk_override(int) {}
void set_attention_tuning(int, int) {}
int attention_fault_flag() { return 0; }
tb_status launch_attention_decode(const AttnArgs&, cudaStream_t) { return absent(); }
tb_status launch_rope_append_rows(const AttnArgs&, cudaStream_t) { return absent(); }
size_t static_attention_scratch_capacity() { return 0; }
tb_status static_attention_scratch(void**) { return absent(); }
int w4_step_grid() { return 0; }
bool w4_step_supports(int64_t, int64_t, int, int) { return false; }
int w4_step_rows_per_stage(int64_t, int, int) { return 0; }
int w4_step_attn_split(int, int) { return 0; }
tb_status launch_w4_step(const StepProgram&, cudaStream_t) { return absent(); }
tb_status launch_w4_step_gemv(const GemvArgs&, cudaStream_t) { return absent(); }
tb_status launch_step_embed(const float*, const int32_t*, const int32_t*, const float*, float*, float*, float*, int32_t*, int64_t, int64_t, int64_t,
                            cudaStream_t) {
  return absent();
}
int step_fault_flag() { return 0; }
void set_step_wait_limit(long long) {}
void set_step_debug(int) {}
tb_status step_wait_probe(long long) { return absent(); }

}  // namespace tb

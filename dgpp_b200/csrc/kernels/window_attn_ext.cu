// Entry points of the grouped attention over a paged cache with convolutions, kept first tokens, caps, sinks, value norms and rotated values
// (kernels: window_attn.cuh).
#include "kernels/window_attn.cuh"

using namespace dgpp;

DGPP_API int dgpp_qk_norm_append_ext(WA_COMMON, int f32, cudaStream_t st) {
  DGPP_REQUIRE(extras != nullptr && maps == 1, "qk_norm_append: this form has extras and one map");
  return wa_append_rows<true>(WA_ARGS, f32, st);
}

DGPP_API int dgpp_window_attn_ext(WA_COMMON, WA_ATTEND) {
  DGPP_REQUIRE(extras != nullptr && maps == 1, "window_attn: this form has extras and one map");
  return wa_attend_rows<true>(WA_ARGS, WA_ATTEND_ARGS);
}

// Entry point of the channel delta rule and of lightning attention (kernels: linear_state.cuh).
#include "kernels/linear_state.cuh"

using namespace dgpp;

// decode = 1: every row is a run of its own; norm and gate are applied (delta) and `out` is written, or the raw read-outs go
// to `o` (lightning).  decode = 0: the runs named by run_start / row_run0, cut into `blocks` = sum of ceil(length / 16) blocks;
// `o` receives the raw read-outs, prep is scratch of rows * (2 hk DK + hv (DV + 3 DK + 1)) + blocks * hv (DK + 512) floats.  delta = 0: lightning (decay [hv]; hk = hv, no low / A_log / dt_bias).
DGPP_API int dgpp_linear_state(const void* proj, int64_t stride, int c_off, int b_off, const void* low, int64_t low_stride,
                               const void* conv_w, void* ring, int taps, const void* A_log, const void* dt_bias, const void* decay,
                               void* state, const void* row_slot, const void* positions, const void* run_start, const void* row_run0,
                               void* prep, void* o, void* out, int64_t out_stride, const void* norm_w, int rows, int runs, int blocks, int hk,
                               int hv, int DK, int DV, int vdim, float q_scale, float eps, int delta, int decode, int f32,
                               cudaStream_t st) {
  LinearArgs a = lin_args(proj, stride, c_off, b_off, conv_w, ring, taps, A_log, dt_bias, state, row_slot, positions, run_start, row_run0,
                          prep, o, rows, runs, blocks, hk, hv, vdim, DV);
  if (lin_check(a, DV, decode)) return -1;
  DGPP_REQUIRE(!delta || (low && A_log && dt_bias), "linear_state: the delta rule needs its decay inputs");
  DGPP_REQUIRE(delta || (decay && hk == hv), "linear_state: lightning needs a decay per head and as many key heads as heads");
  DGPP_REQUIRE(!decode || (delta ? (out && norm_w) : (o != nullptr)), "linear_state: no output");
  if (rows == 0) return 0;
  a.low = static_cast<const float*>(low); a.low_stride = low_stride;
  a.decay = static_cast<const float*>(decay);
  a.out = out; a.out_stride = out_stride; a.norm_w = static_cast<const float*>(norm_w);
  a.q_scale = q_scale; a.eps = eps;
  if (f32) return delta ? launch_lin_dims<float, kDelta>(a, DK, DV, decode, st) : launch_lin_dims<float, kLightning>(a, DK, DV, decode, st);
  return delta ? launch_lin_dims<bf16, kDelta>(a, DK, DV, decode, st) : launch_lin_dims<bf16, kLightning>(a, DK, DV, decode, st);
}

// Entry point of the delta rule with one decay per token and head (kernels: linear_state.cuh).
#include "kernels/linear_state.cuh"

using namespace dgpp;

// Columns of a projection row: q | k | v channels from c_off, raw strengths [hv] from b_off, raw decays [hv] from a_off, raw output
// gates [hv * DV] from g_off.  decode = 1: every row is a run of its own; norm and gate are applied and `out` is written.  decode = 0:
// the runs named by run_start / row_run0, cut into `blocks` = sum of ceil(length / 16) blocks; `o` [rows, hv * DV] receives the raw
// read-outs, prep is scratch of rows * (2 hk DK + hv (DV + 2)) + blocks * hv * 576 floats.
DGPP_API int dgpp_gated_delta(const void* proj, int64_t stride, int c_off, int b_off, int a_off, int g_off, const void* conv_w, void* ring, int taps,
                              const void* A_log, const void* dt_bias, void* state, const void* row_slot, const void* positions,
                              const void* run_start, const void* row_run0, void* prep, void* o, void* out, int64_t out_stride,
                              const void* norm_w, int rows, int runs, int blocks, int hk, int hv, int DK, int DV, int vdim, float q_scale,
                              float eps, int decode, int f32, cudaStream_t st) {
  LinearArgs a = lin_args(proj, stride, c_off, b_off, conv_w, ring, taps, A_log, dt_bias, state, row_slot, positions, run_start, row_run0,
                          prep, o, rows, runs, blocks, hk, hv, vdim, DV);
  if (lin_check(a, DV, decode)) return -1;
  DGPP_REQUIRE(A_log && dt_bias && conv_w, "gated_delta: the rule needs its convolution and decay inputs");
  DGPP_REQUIRE(!decode || (out && norm_w), "gated_delta: no output");
  if (rows == 0) return 0;
  a.a_off = a_off; a.g_off = g_off;
  a.out = out; a.out_stride = out_stride; a.norm_w = static_cast<const float*>(norm_w);
  a.q_scale = q_scale; a.eps = eps;
  return f32 ? launch_lin_dims<float, kScalarDelta>(a, DK, DV, decode, st) : launch_lin_dims<bf16, kScalarDelta>(a, DK, DV, decode, st);
}

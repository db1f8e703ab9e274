// Entry point of the state-space recurrence with scalar decays (Mamba-2 form; kernels: linear_state.cuh).
#include "kernels/linear_state.cuh"

using namespace dgpp;

// proj: conv channels q [hk, DK] | k [hk, DK] | v [hv, DV] from column c_off, raw step sizes [hv] at b_off.  Read-outs go to `o`
// [rows, hv * vdim] fp32.  decode = 1: every row is a run of its own.  decode = 0: the runs named by run_start / row_run0, cut
// into `blocks` = sum of ceil(length / 16) blocks; prep is scratch of rows * (2 hk DK + hv (DV + 2)) + blocks * hv * 288 floats.
DGPP_API int dgpp_state_space(const void* proj, int64_t stride, int c_off, int b_off, const void* conv_w, const void* conv_b, void* ring,
                              int taps, const void* A_log, const void* dt_bias, const void* skip, void* state, const void* row_slot,
                              const void* positions, const void* run_start, const void* row_run0, void* prep, void* o, int rows,
                              int runs, int blocks, int hk, int hv, int DK, int DV, int vdim, int decode, int f32, cudaStream_t st) {
  LinearArgs a = lin_args(proj, stride, c_off, b_off, conv_w, ring, taps, A_log, dt_bias, state, row_slot, positions, run_start, row_run0,
                          prep, o, rows, runs, blocks, hk, hv, vdim, vdim);
  if (lin_check(a, DV, decode)) return -1;
  DGPP_REQUIRE(A_log && dt_bias && skip && o && conv_w, "state_space: A_log, dt_bias, skip, the convolution and an output are required");
  if (rows == 0) return 0;
  a.conv_b = static_cast<const float*>(conv_b);
  a.skip = static_cast<const float*>(skip);
  return f32 ? launch_lin_dims<float, kStateSpace>(a, DK, DV, decode, st) : launch_lin_dims<bf16, kStateSpace>(a, DK, DV, decode, st);
}

// Entry point of the matrix memory with exponential gates (the mLSTM of xLSTM; kernels: linear_state.cuh).
#include "kernels/linear_state.cuh"

using namespace dgpp;

// Columns of a projection row: q | k [hv * DK] | v [hv * DV] from c_off, raw input gates [hv] from i_off, raw forget gates [hv] from f_off,
// raw output gates [hv * DV] from g_off.  nstate [slots, hv, DK + 4].  decode = 1: every row is a run of its own; norm (norm_w [hv * DV])
// and gate are applied and `out` is written.  decode = 0: the runs named by run_start / row_run0, cut into `blocks` = sum of
// ceil(length / 16) blocks; `o` [rows, hv * DV] receives the raw read-outs, `den` [rows, hv] what they are to be divided by; prep is scratch
// of rows * hv * (2 DK + DV + 3) + blocks * hv * 288 floats.
DGPP_API int dgpp_matrix_memory(const void* proj, int64_t stride, int c_off, int i_off, int f_off, int g_off, const void* i_bias, const void* f_bias,
                                float gate_cap, void* state, void* nstate, const void* row_slot, const void* positions, const void* run_start,
                                const void* row_run0, void* prep, void* o, void* den, void* out, int64_t out_stride, const void* norm_w, int rows,
                                int runs, int blocks, int hv, int DK, int DV, int vdim, float q_scale, float eps, int decode, int f32, cudaStream_t st) {
  LinearArgs a = lin_args(proj, stride, c_off, i_off, nullptr, nullptr, 0, nullptr, nullptr, state, row_slot, positions, run_start, row_run0, prep, o,
                          rows, runs, blocks, hv, hv, vdim, DV);
  if (lin_check(a, DV, decode)) return -1;
  DGPP_REQUIRE(i_bias && f_bias && nstate && gate_cap > 0.f, "matrix_memory: gate biases, a cap and the norm's state are required");
  DGPP_REQUIRE(stride % 4 == 0 && c_off % 4 == 0, "matrix_memory: unaligned projection rows");
  DGPP_REQUIRE(decode ? (out && norm_w) : den != nullptr, "matrix_memory: no output");
  if (rows == 0) return 0;
  a.a_off = f_off; a.g_off = g_off;
  a.i_bias = static_cast<const float*>(i_bias); a.f_bias = static_cast<const float*>(f_bias); a.gate_cap = gate_cap;
  a.nstate = static_cast<float*>(nstate); a.den = static_cast<float*>(den);
  a.out = out; a.out_stride = out_stride; a.norm_w = static_cast<const float*>(norm_w);
  a.q_scale = q_scale; a.eps = eps;
  return f32 ? launch_lin_dims<float, kMatrix>(a, DK, DV, decode, st) : launch_lin_dims<bf16, kMatrix>(a, DK, DV, decode, st);
}

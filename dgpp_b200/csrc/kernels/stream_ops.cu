// Row operators of models that keep the residual stream in fp32 (activations T = bf16 or fp32):
//   embed_rows        out[r] = table[ids[r]]                                                   (fp32 rows)
//   resid_norm        x += delta (fp32, optional); out = x / sqrt(mean(x^2) + eps) * w           (out in T)
//   gated_group_norm  per group of columns: out = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate) * scale
//   geglu             out = gelu_tanh(gate) * up
// Rows may carry zero columns behind their `n` true ones (the padding of the tensor-core GEMM): means divide by the true
// count and the padded columns stay zero.  Norms, gates and the sum are fp32; one rounding to T at the end.
#include <math.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

constexpr int kStreamThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kStreamThreads)
embed_rows_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int cols, int vocab) {
  pdl_wait();
  const int row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + static_cast<size_t>(id) * cols;
  float* dst = out + static_cast<size_t>(row) * cols;
  for (int i = threadIdx.x * 4; i < cols; i += kStreamThreads * 4) st_elem4(dst + i, ld_elem4(src + i));
}

template <typename T>
__global__ void __launch_bounds__(kStreamThreads)
resid_norm_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ w, T* __restrict__ out,
                  int cols, int n, float eps) {
  __shared__ float scratch[kStreamThreads / 32];
  pdl_wait();
  const size_t base = static_cast<size_t>(blockIdx.x) * cols;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < cols; i += kStreamThreads * 4) {
    float4 v = ld_elem4(x + base + i);
    if (delta != nullptr) {
      const float4 d = ld_elem4(delta + base + i);
      v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
      st_elem4(x + base + i, v);
    }
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float r = 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(n) + eps);
  for (int i = threadIdx.x * 4; i < cols; i += kStreamThreads * 4) {
    const float4 v = ld_elem4(x + base + i), g = ld_elem4(w + i);
    st_elem4(out + base + i, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
  }
}

// o [rows, groups * gp] fp32, gate [rows, gate_stride] (TG), w [gp] shared by the groups.  A group is handled by `team` threads
// (a warp, or the whole CTA for wide groups).
template <typename T, typename TG>
__global__ void __launch_bounds__(kStreamThreads)
gated_group_norm_kernel(const float* __restrict__ o, const TG* __restrict__ gate, int64_t gate_stride, const float* __restrict__ w,
                        T* __restrict__ out, int64_t out_stride, int rows, int groups, int gp, int n, float eps, float scale, int team) {
  __shared__ float scratch[kStreamThreads / 32];
  pdl_wait();
  const size_t unit = (static_cast<size_t>(blockIdx.x) * kStreamThreads + threadIdx.x) / team;
  const bool live = unit < static_cast<size_t>(rows) * groups;
  const int me = threadIdx.x % team;
  const size_t row = live ? unit / groups : 0;
  const int g = live ? static_cast<int>(unit % groups) : 0;
  const float* op = o + (row * groups + g) * static_cast<size_t>(gp);
  const TG* gt = gate + row * gate_stride + static_cast<size_t>(g) * gp;
  T* dst = out + row * out_stride + static_cast<size_t>(g) * gp;
  float ss = 0.f;
  for (int i = me * 4; i < gp; i += team * 4) {
    const float4 v = ld_elem4(op + i);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = team == 32 ? warp_sum_f32(ss) : block_sum_f32(ss, scratch);
  if (!live) return;
  const float r = scale / sqrtf(ss / static_cast<float>(n) + eps);
  for (int i = me * 4; i < gp; i += team * 4) {
    const float4 v = ld_elem4(op + i), a = ld_elem4(gt + i), ww = ld_elem4(w + i);
    st_elem4(dst + i, make_float4(v.x * r * ww.x * sigmoid_f32(a.x), v.y * r * ww.y * sigmoid_f32(a.y),
                                  v.z * r * ww.z * sigmoid_f32(a.z), v.w * r * ww.w * sigmoid_f32(a.w)));
  }
}

// 0.5 z (1 + tanh(u)) = z / (1 + exp(-2 u)),  u = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_f32(float z) {
  return z / (1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

// gate_up [rows, 2 * inter] (gate columns, then up columns) -> out [rows, inter]
template <typename T>
__global__ void __launch_bounds__(kStreamThreads)
geglu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter) {
  pdl_wait();
  const size_t row = blockIdx.y;
  const int i = (blockIdx.x * kStreamThreads + threadIdx.x) * 4;
  if (i >= inter) return;
  const float4 g = ld_elem4(gate_up + row * 2 * inter + i), u = ld_elem4(gate_up + row * 2 * inter + inter + i);
  st_elem4(out + row * inter + i, make_float4(gelu_tanh_f32(g.x) * u.x, gelu_tanh_f32(g.y) * u.y,
                                              gelu_tanh_f32(g.z) * u.z, gelu_tanh_f32(g.w) * u.w));
}

}  // namespace dgpp

using namespace dgpp;

// `f32` selects fp32 activations (else bf16) in every entry point below.
DGPP_API int dgpp_embed_rows(const void* ids, const void* table, void* out, int rows, int cols, int vocab, int f32, cudaStream_t st) {
  DGPP_REQUIRE(cols % 8 == 0, "embed_rows: %d columns (a multiple of 8)", cols);
  if (rows == 0) return 0;
  if (f32) embed_rows_kernel<float><<<rows, kStreamThreads, 0, st>>>(static_cast<const int32_t*>(ids), static_cast<const float*>(table), static_cast<float*>(out), cols, vocab);
  else embed_rows_kernel<bf16><<<rows, kStreamThreads, 0, st>>>(static_cast<const int32_t*>(ids), static_cast<const bf16*>(table), static_cast<float*>(out), cols, vocab);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

DGPP_API int dgpp_resid_norm(void* x, const void* delta, const void* w, void* out, int rows, int cols, int n, float eps, int f32, cudaStream_t st) {
  DGPP_REQUIRE(cols % 8 == 0 && n >= 1 && n <= cols, "resid_norm: %d of %d columns", n, cols);
  if (rows == 0) return 0;
  float* xp = static_cast<float*>(x);
  const float *dp = static_cast<const float*>(delta), *wp = static_cast<const float*>(w);
  if (f32) resid_norm_kernel<float><<<rows, kStreamThreads, 0, st>>>(xp, dp, wp, static_cast<float*>(out), cols, n, eps);
  else resid_norm_kernel<bf16><<<rows, kStreamThreads, 0, st>>>(xp, dp, wp, static_cast<bf16*>(out), cols, n, eps);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// gate_f32: the gate rows are fp32 although the activations are bf16.
DGPP_API int dgpp_gated_group_norm(const void* o, const void* gate, int64_t gate_stride, const void* w, void* out, int64_t out_stride,
                                   int rows, int groups, int gp, int n, float eps, float scale, int f32, int gate_f32, cudaStream_t st) {
  DGPP_REQUIRE(gp % 8 == 0 && gate_stride % 8 == 0 && out_stride % 8 == 0 && n >= 1 && n <= gp, "gated_group_norm: %d of %d columns", n, gp);
  if (rows == 0) return 0;
  const int team = gp <= 512 ? 32 : kStreamThreads;
  const int64_t blocks = dgpp_ceil_div64(static_cast<int64_t>(rows) * groups * team, kStreamThreads);
  const float *op = static_cast<const float*>(o), *wp = static_cast<const float*>(w);
#define DGPP_GGN(TT, TG) gated_group_norm_kernel<TT, TG><<<static_cast<unsigned>(blocks), kStreamThreads, 0, st>>>( \
      op, static_cast<const TG*>(gate), gate_stride, wp, static_cast<TT*>(out), out_stride, rows, groups, gp, n, eps, scale, team)
  if (f32) DGPP_GGN(float, float);
  else if (gate_f32) DGPP_GGN(bf16, float);
  else DGPP_GGN(bf16, bf16);
#undef DGPP_GGN
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

DGPP_API int dgpp_geglu(const void* gate_up, void* out, int rows, int inter, int f32, cudaStream_t st) {
  DGPP_REQUIRE(inter % 8 == 0, "geglu: width %d (a multiple of 8)", inter);
  if (rows == 0) return 0;
  DGPP_REQUIRE(rows <= 65535, "geglu: %d rows", rows);
  const dim3 grid(dgpp_ceil_div(inter / 4, kStreamThreads), rows);
  if (f32) geglu_kernel<float><<<grid, kStreamThreads, 0, st>>>(static_cast<const float*>(gate_up), static_cast<float*>(out), inter);
  else geglu_kernel<bf16><<<grid, kStreamThreads, 0, st>>>(static_cast<const bf16*>(gate_up), static_cast<bf16*>(out), inter);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

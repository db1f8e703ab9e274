// Entry points of the grouped attention over a paged cache, plain form (kernels: window_attn.cuh), and the combination of the two maps of
// differential attention.
#include "kernels/window_attn.cuh"

namespace dgpp {

struct DiffCombine {
  const float* ml;          // [n, 2 heads, splits, 2], or null: acc holds finished outputs [rows, 2 heads, DV]
  const float* acc;         // [n, 2 heads, splits, DV]
  const void* gate;         // [rows, gate_stride] (T), column h * DV + d
  int64_t gate_stride;
  void* out;                // [rows, out_stride] (T)
  int64_t out_stride;
  const int32_t* row_list;
  int n, heads, group, vdim, splits;
  float lambda, factor, eps;
};

// One warp per (row, output head), four warps per CTA; value columns 2 * lane + 64 * j.
template <typename T, int NV>
__global__ void __launch_bounds__(128) diff_combine_kernel(DiffCombine p) {
  constexpr int DV = NV * 64;
  pdl_wait();
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= p.n * p.heads) return;
  const int i = unit / p.heads, h = unit % p.heads, row = p.row_list ? p.row_list[i] : i;
  float2 o[NV];
#pragma unroll
  for (int map = 0; map < 2; ++map) {
    const size_t rh = static_cast<size_t>(p.ml != nullptr ? i : row) * 2 * p.heads + (h / p.group * 2 + map) * p.group + h % p.group;
    float2 a[NV];
#pragma unroll
    for (int j = 0; j < NV; ++j) a[j] = make_float2(0.f, 0.f);
    float mm = -INFINITY, ll = 0.f;
    if (p.ml != nullptr)
      for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.ml[(rh * p.splits + s) * 2]);
    for (int s = 0; s < p.splits; ++s) {
      float c = 1.f;
      if (p.ml != nullptr) {
        const float ms = p.ml[(rh * p.splits + s) * 2];
        c = ms == -INFINITY ? 0.f : wa_exp<T>(ms - mm);
        ll += p.ml[(rh * p.splits + s) * 2 + 1] * c;
      }
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const float2 v = *reinterpret_cast<const float2*>(p.acc + (rh * p.splits + s) * DV + 64 * j + 2 * lane);
        a[j].x = fmaf(v.x, c, a[j].x);
        a[j].y = fmaf(v.y, c, a[j].y);
      }
    }
    const float r = p.ml == nullptr ? 1.f : (ll > 0.f ? 1.f / ll : 0.f), f = map ? -p.lambda * r : r;
#pragma unroll
    for (int j = 0; j < NV; ++j) o[j] = map ? make_float2(fmaf(a[j].x, f, o[j].x), fmaf(a[j].y, f, o[j].y)) : make_float2(a[j].x * f, a[j].y * f);
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) ss = fmaf(o[j].x, o[j].x, fmaf(o[j].y, o[j].y, ss));
  const float r = p.factor / sqrtf(warp_sum_f32(ss) / static_cast<float>(p.vdim) + p.eps);
  const T* gate = static_cast<const T*>(p.gate) + row * p.gate_stride + static_cast<size_t>(h) * DV + 2 * lane;
  T* dst = static_cast<T*>(p.out) + row * p.out_stride + static_cast<size_t>(h) * DV + 2 * lane;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const float2 g = ld_elem2(gate + 64 * j);
    st_elem(dst + 64 * j, o[j].x * r * sigmoid_f32(g.x));
    st_elem(dst + 64 * j + 1, o[j].y * r * sigmoid_f32(g.y));
  }
}

}  // namespace dgpp

using namespace dgpp;

DGPP_API int dgpp_qk_norm_append(WA_COMMON, int f32, cudaStream_t st) {
  DGPP_REQUIRE(extras == nullptr, "qk_norm_append: the plain form has no extras");
  return wa_append_rows<false>(WA_ARGS, f32, st);
}

DGPP_API int dgpp_window_attn(WA_COMMON, WA_ATTEND) {
  DGPP_REQUIRE(extras == nullptr, "window_attn: the plain form has no extras");
  return wa_attend_rows<false>(WA_ARGS, WA_ATTEND_ARGS);
}

// out[row, h] = rms-normed (a1 - lambda a2) * factor * sigmoid(gate) for n rows (row_list names them when given) of `heads` output
// heads, `group` per kv head; ml null: acc holds finished outputs of all rows of the pass (one split).
DGPP_API int dgpp_diff_combine(const void* ml, const void* acc, const void* gate, int64_t gate_stride, const void* row_list, void* out,
                               int64_t out_stride, int n, int heads, int group, int DV, int vdim, int splits, float lambda, float factor, float eps,
                               int f32, cudaStream_t st) {
  DGPP_REQUIRE(DV % 64 == 0 && DV >= 64 && DV <= 256 && vdim >= 1 && vdim <= DV && group >= 1 && heads % group == 0 && splits >= 1 && (ml || splits == 1),
               "diff_combine: %d heads of %d columns, %d splits", heads, DV, splits);
  if (n == 0) return 0;
  const DiffCombine p = {static_cast<const float*>(ml), static_cast<const float*>(acc), gate, gate_stride, out, out_stride,
                         static_cast<const int32_t*>(row_list), n, heads, group, vdim, splits, lambda, factor, eps};
  const int64_t grid = dgpp_ceil_div64(static_cast<int64_t>(n) * heads, 4);
#define DGPP_DC(NV) if (DV == NV * 64) { if (f32) diff_combine_kernel<float, NV><<<static_cast<unsigned>(grid), 128, 0, st>>>(p); \
                                         else diff_combine_kernel<bf16, NV><<<static_cast<unsigned>(grid), 128, 0, st>>>(p); }
  DGPP_DC(1) DGPP_DC(2) DGPP_DC(3) DGPP_DC(4)
#undef DGPP_DC
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// Causal depthwise convolution over time on the columns of projection rows (T = bf16 or fp32), for passes over runs of consecutive tokens:
//
//   u_t = x_t + bias,   y_t = sum_j w[j] u_(t - taps + 1 + j)      (fp32; one rounding to T; zeros before the request's first token)
//
//   short_conv   a thread owns four channels of 16 rows and slides the window along in registers (up to four taps; more taps reread the
//                rows); inputs before the run's first row come from the request's ring
//   conv_tail    the newest inputs of every run go to the ring, once every reader is done
//
// The ring holds `taps` inputs per channel and request (fp32, bias included), entry p % taps for position p: see window_attn.cuh, whose
// decode form convolves single tokens itself.
#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

struct ShortConv {
  const void* x;             // [rows, stride]
  int64_t stride;
  const float* bias;         // [C] or null
  const float* w;            // [taps, C] (last row: the current token)
  float* ring;               // [requests, taps, C]
  const int32_t* row_req;    // [rows]
  const int32_t* positions;  // [rows]
  const int32_t* row_run0;   // [rows] first row of the row's run
  const int32_t* run_start;  // [runs + 1]
  void* out;                 // [rows, C]
  int rows, C, taps;
};

constexpr int kConvRows = 16;

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 mad4(float4 w, float4 u, float4 a) {
  return make_float4(fmaf(w.x, u.x, a.x), fmaf(w.y, u.y, a.y), fmaf(w.z, u.z, a.z), fmaf(w.w, u.w, a.w));
}

// The input j rows before `row` (position pos, `back` rows into its run), bias added.
template <typename T>
__device__ __forceinline__ float4 conv_past(const ShortConv& p, const T* x, float4 bias, int row, int pos, int back, int j, int ch) {
  if (j > pos) return make_float4(0.f, 0.f, 0.f, 0.f);
  if (j <= back) return add4(ld_elem4(x + static_cast<int64_t>(row - j) * p.stride), bias);
  return ld_elem4(p.ring + (static_cast<size_t>(p.row_req[row]) * p.taps + (pos - j) % p.taps) * p.C + ch);
}

// grid (ceil(C / 512), ceil(rows / 16)), 128 threads.  TAPS 0: any number, window not kept.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(ShortConv p) {
  pdl_wait();
  const int ch = (blockIdx.x * 128 + threadIdx.x) * 4, r0 = blockIdx.y * kConvRows;
  if (ch >= p.C) return;
  const int n = min(kConvRows, p.rows - r0);
  const T* x = static_cast<const T*>(p.x) + ch;
  T* out = static_cast<T*>(p.out) + ch;
  const float4 bias = p.bias != nullptr ? ld_elem4(p.bias + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
  if (TAPS == 0) {
    for (int k = 0; k < n; ++k) {
      const int row = r0 + k, pos = p.positions[row], back = row - p.row_run0[row];
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = p.taps - 1; j >= 0; --j)
        acc = mad4(ld_elem4(p.w + static_cast<size_t>(p.taps - 1 - j) * p.C + ch), conv_past(p, x, bias, row, pos, back, j, ch), acc);
      st_elem4(out + static_cast<size_t>(row) * p.C, acc);
    }
    return;
  }
  constexpr int N = TAPS > 0 ? TAPS : 1;
  float4 w[N], h[N];                                       // h[j]: the input j tokens back
#pragma unroll
  for (int j = 0; j < N; ++j) w[j] = ld_elem4(p.w + static_cast<size_t>(N - 1 - j) * p.C + ch);
#pragma unroll 4
  for (int k = 0; k < n; ++k) {
    const int row = r0 + k, run0 = p.row_run0[row];
    if (k == 0 || run0 == row) {                           // a window that this thread has not seen
      const int pos = p.positions[row];
#pragma unroll
      for (int j = 1; j < N; ++j) h[j] = conv_past(p, x, bias, row, pos, row - run0, j, ch);
    }
    h[0] = add4(ld_elem4(x + static_cast<int64_t>(row) * p.stride), bias);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < N; ++j) acc = mad4(w[j], h[j], acc);
    st_elem4(out + static_cast<size_t>(row) * p.C, acc);
#pragma unroll
    for (int j = N - 1; j > 0; --j) h[j] = h[j - 1];
  }
}

// grid (ceil(C / 1024), runs)
template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(ShortConv p) {
  pdl_wait();
  const int ch = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (ch >= p.C) return;
  const int first = p.run_start[blockIdx.y], last = p.run_start[blockIdx.y + 1];
  const float4 bias = p.bias != nullptr ? ld_elem4(p.bias + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
  for (int row = max(first, last - p.taps); row < last; ++row)
    st_elem4(p.ring + (static_cast<size_t>(p.row_req[row]) * p.taps + p.positions[row] % p.taps) * p.C + ch,
             add4(ld_elem4(static_cast<const T*>(p.x) + static_cast<int64_t>(row) * p.stride + ch), bias));
}

template <typename T>
static int launch_short_conv(const ShortConv& p, int runs, cudaStream_t st) {
  const dim3 grid(dgpp_ceil_div(p.C, 512), dgpp_ceil_div(p.rows, kConvRows));
  if (p.taps == 1) short_conv_kernel<T, 1><<<grid, 128, 0, st>>>(p);
  else if (p.taps == 2) short_conv_kernel<T, 2><<<grid, 128, 0, st>>>(p);
  else if (p.taps == 3) short_conv_kernel<T, 3><<<grid, 128, 0, st>>>(p);
  else if (p.taps == 4) short_conv_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else short_conv_kernel<T, 0><<<grid, 128, 0, st>>>(p);
  DGPP_CUDA_OK(cudaGetLastError());
  conv_tail_kernel<T><<<dim3(dgpp_ceil_div(p.C, 1024), runs), 256, 0, st>>>(p);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

}  // namespace dgpp

using namespace dgpp;

// x [rows, stride] -> out [rows, C] (T); runs of consecutive rows, one per request: run_start [runs + 1], row_run0 [rows].  The ring
// takes in the runs' newest inputs.
DGPP_API int dgpp_short_conv(const void* x, int64_t stride, const void* bias, const void* w, void* ring, const void* row_req, const void* positions,
                             const void* row_run0, const void* run_start, void* out, int rows, int runs, int C, int taps, int f32, cudaStream_t st) {
  DGPP_REQUIRE(C >= 4 && C % 4 == 0 && stride % 4 == 0 && taps >= 1, "short_conv: %d channels, %d taps", C, taps);
  DGPP_REQUIRE(rows >= 0 && rows <= 65535 * kConvRows && runs >= 0 && runs <= 65535, "short_conv: %d rows in %d runs", rows, runs);
  if (rows == 0) return 0;
  const ShortConv p = {x, stride, static_cast<const float*>(bias), static_cast<const float*>(w), static_cast<float*>(ring),
                       static_cast<const int32_t*>(row_req), static_cast<const int32_t*>(positions), static_cast<const int32_t*>(row_run0),
                       static_cast<const int32_t*>(run_start), out, rows, C, taps};
  return f32 ? launch_short_conv<float>(p, runs, st) : launch_short_conv<bf16>(p, runs, st);
}

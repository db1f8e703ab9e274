// True fp32 linear layer on the CUDA cores:  C[T, N] = alpha * X[T, K] . W[N, K]^T, fp32 multiply-adds, K in ascending
// order (no reduced-precision tensor mode), so a row's result depends only on that row.  The 32-bit twin of the tcgen05
// GEMM for models that run in fp32.  The grouped form multiplies every tile of `bn` rows by its own matrix out of a stack.
#include "common/common.h"
#include "common/ptx.cuh"

namespace dgpp {

constexpr int kGfTile = 64, kGfK = 16, kGfThreads = 256;

__global__ void __launch_bounds__(kGfThreads)
gemm_f32_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ w, float alpha, float* __restrict__ out,
                int64_t ldc, int T, int N, int K, const int32_t* __restrict__ groups, int bn, int group_x) {
  __shared__ __align__(16) float xs[kGfK][kGfTile + 4], ws[kGfK][kGfTile + 4];
  pdl_wait();
  const int n0 = blockIdx.x * kGfTile, tid = threadIdx.x;
  int m0 = blockIdx.y * kGfTile;
  if (groups != nullptr) {                                 // tile blockIdx.y: T = its row count, x / out / w start at its own rows
    const int e = groups[blockIdx.y];
    if (e < 0) return;
    m0 = 0;
    T = group_x ? bn : min(T, bn);
    w += static_cast<size_t>(e) * N * K;
    if (group_x) x += static_cast<size_t>(blockIdx.y) * bn * ldx;
    out += static_cast<size_t>(blockIdx.y) * bn * ldc;
  }
  const int tx = tid % 16, ty = tid / 16;
  const int lr = tid / 4, lk = (tid % 4) * 4;              // staging: row of the tile, 4 consecutive k
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kGfK) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (k0 + lk < K) {                                     // K is a multiple of 4
      if (m0 + lr < T) a = *reinterpret_cast<const float4*>(x + static_cast<size_t>(m0 + lr) * ldx + k0 + lk);
      if (n0 + lr < N) b = *reinterpret_cast<const float4*>(w + static_cast<size_t>(n0 + lr) * K + k0 + lk);
    }
    __syncthreads();
    xs[lk][lr] = a.x; xs[lk + 1][lr] = a.y; xs[lk + 2][lr] = a.z; xs[lk + 3][lr] = a.w;
    ws[lk][lr] = b.x; ws[lk + 1][lr] = b.y; ws[lk + 2][lr] = b.z; ws[lk + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kGfK; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float am[4] = {av.x, av.y, av.z, av.w}, bm[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(am[i], bm[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= T) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) out[static_cast<size_t>(m) * ldc + n] = acc[i][j] * alpha;
    }
  }
}

}  // namespace dgpp

using namespace dgpp;

DGPP_API int dgpp_gemm_f32(const void* x, int64_t ldx, const void* w, float alpha, void* out, int64_t ldc, int T, int N, int K, cudaStream_t st) {
  DGPP_REQUIRE(T >= 1 && N >= 1, "gemm_f32: empty problem");
  DGPP_REQUIRE(K % 4 == 0 && ldx % 4 == 0, "gemm_f32: K %d / row stride %lld must be multiples of 4", K, static_cast<long long>(ldx));
  const dim3 grid(dgpp_ceil_div(N, kGfTile), dgpp_ceil_div(T, kGfTile));
  DGPP_REQUIRE(grid.y <= 65535, "gemm_f32: %d rows", T);
  gemm_f32_kernel<<<grid, kGfThreads, 0, st>>>(static_cast<const float*>(x), ldx, static_cast<const float*>(w), alpha, static_cast<float*>(out), ldc, T, N, K, nullptr, 0, 0);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// See dgpp_gemm_tc_grouped.
DGPP_API int dgpp_gemm_f32_grouped(int bn, const void* x, int64_t ldx, int x_rows, int group_x, const void* w, int experts, const void* groups,
                                   void* out, int64_t ldc, int tiles, int N, int K, cudaStream_t st) {
  DGPP_REQUIRE(groups != nullptr && experts >= 1 && tiles >= 1 && tiles <= 65535, "gemm_f32_grouped: %d tiles over %d matrices", tiles, experts);
  DGPP_REQUIRE(bn >= 1 && bn <= kGfTile && (group_x ? x_rows == tiles * bn : (x_rows >= 1 && x_rows <= bn)),
               "gemm_f32_grouped: %d rows in %d tiles of %d", x_rows, tiles, bn);
  DGPP_REQUIRE(K % 4 == 0 && ldx % 4 == 0, "gemm_f32_grouped: K %d / row stride %lld must be multiples of 4", K, static_cast<long long>(ldx));
  gemm_f32_kernel<<<dim3(dgpp_ceil_div(N, kGfTile), tiles), kGfThreads, 0, st>>>(
      static_cast<const float*>(x), ldx, static_cast<const float*>(w), 1.f, static_cast<float*>(out), ldc, x_rows, N, K,
      static_cast<const int32_t*>(groups), bn, group_x);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

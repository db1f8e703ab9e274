// Element access shared by kernels that exist for 16-bit and for true 32-bit activations: scalar and vector loads /
// stores that convert to and from fp32 registers.
#pragma once
#include "common/dtypes.cuh"

namespace dgpp {

__device__ __forceinline__ float ld_elem(const bf16* p) { return bf16_to_f32(*p); }
__device__ __forceinline__ float ld_elem(const float* p) { return *p; }
__device__ __forceinline__ void st_elem(bf16* p, float v) { *p = f32_to_bf16(v); }
__device__ __forceinline__ void st_elem(float* p, float v) { *p = v; }

// Two consecutive elements (8-byte aligned for fp32, 4-byte for bf16).
__device__ __forceinline__ float2 ld_elem2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const bf162*>(p)); }
__device__ __forceinline__ float2 ld_elem2(const float* p) { return *reinterpret_cast<const float2*>(p); }

// Four consecutive elements (16-byte aligned for fp32, 8-byte for bf16).
__device__ __forceinline__ float4 ld_elem4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld_elem4(const bf16* p) {
  const uint2 w = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&w.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&w.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st_elem4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st_elem4(bf16* p, float4 v) {
  bf162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 w;
  w.x = *reinterpret_cast<uint32_t*>(&a);
  w.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = w;
}

// Eight consecutive elements (16-byte aligned).
__device__ __forceinline__ void ld_elem8(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void ld_elem8(const bf16* p, float* f) {
  Pack16 v;
  v.u = *reinterpret_cast<const uint4*>(p);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 t = __bfloat1622float2(v.h2[j]);
    f[2 * j] = t.x;
    f[2 * j + 1] = t.y;
  }
}
__device__ __forceinline__ void st_elem8(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void st_elem8(bf16* p, const float* f) {
  Pack16 v;
#pragma unroll
  for (int j = 0; j < 4; ++j) v.h2[j] = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
  *reinterpret_cast<uint4*>(p) = v.u;
}

// 16 bytes of elements: 8 bf16 or 4 fp32, converted to fp32.
template <typename T>
struct Vec16;
template <>
struct Vec16<bf16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    Pack16 v;
    v.u = *reinterpret_cast<const uint4*>(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 t = __bfloat1622float2(v.h2[j]);
      f[2 * j] = t.x;
      f[2 * j + 1] = t.y;
    }
  }
};
template <>
struct Vec16<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
};

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float warp_sum_f32(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the CTA in a fixed order (lanes by xor-tree, warps ascending); scratch: one float per warp.
__device__ __forceinline__ float block_sum_f32(float v, float* scratch) {
  v = warp_sum_f32(v);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  const int nw = blockDim.x >> 5;
  for (int i = 0; i < nw; ++i) t += scratch[i];
  __syncthreads();
  return t;
}

// 16-byte asynchronous copy global -> shared.
__device__ __forceinline__ void cp_async_16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_group_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_group_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace dgpp

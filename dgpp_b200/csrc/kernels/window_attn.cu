// Sliding-window GQA over a paged cache of 16-bit or true 32-bit keys and values, with per-head query / key norms, no
// rotation, a softmax scale of its own and value heads that may be wider or narrower than the key heads.
//
//   query head h reads key/value head g = h / (hq / hkv);  qn = rms(q_h) * wq, kn = rms(k_g) * wk (fp32)
//   row at position i attends to positions max(0, i - window + 1) .. i:  p = softmax(scale * qn . kn),  out = sum p v
//
// The projections of a row sit in one fused row (T = bf16 or fp32); head widths are padded to multiples of 64 with zero
// columns (D for queries / keys, DV for values), `dim` is the true key width that the norms divide by.
// Cache: k [blocks, hkv, page, D], v [blocks, hkv, page, DV].
//
//   qk_norm_append   prompt rows: norms q in place, appends normed k and v to the cache (one warp per row and head)
//   window_attn      one (row, kv head, split of the window) per CTA; `fused` = every row is the newest token of its
//                    request and the CTA norms q, norms and appends k / v itself (decode: one launch per layer)
// Softmax statistics and sums are fp32; the partials of the splits merge in ascending order.
#include <math.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

struct WindowAttnParams {
  void* proj;               // [rows, stride]: q heads at q_off + h * D, k heads at k_off + g * D, v heads at v_off + g * DV
  int64_t stride;
  int q_off, k_off, v_off;
  const float* wq;          // [D] fp32 norm weights (zero beyond dim)
  const float* wk;
  void* k_cache;
  void* v_cache;
  const int32_t* block_table;
  const int32_t* row_req;
  const int32_t* positions;
  const int32_t* row_list;  // optional: the rows of this launch (else 0 .. grid - 1)
  float* part_ml;           // [rows, hq, splits, 2]   (splits > 1)
  float* part_acc;          // [rows, hq, splits, DV]
  void* out;                // [rows, out_stride] head h at column h * DV
  int64_t out_stride;
  int hq, hkv, D, DV, dim, page, max_blocks, splits, window, fused;
  float scale, eps, out_scale;
};

constexpr int kWaWarps = 4;

template <typename T>
__device__ __forceinline__ float wa_exp(float x);
template <>
__device__ __forceinline__ float wa_exp<float>(float x) { return expf(x); }
template <>
__device__ __forceinline__ float wa_exp<bf16>(float x) { return __expf(x); }

__device__ __forceinline__ size_t wa_token(const WindowAttnParams& p, const int32_t* bt, int g, int t) {
  return (static_cast<size_t>(bt[t / p.page]) * p.hkv + g) * p.page + t % p.page;
}

// 1 / rms of one head, by one warp
template <typename T>
__device__ __forceinline__ float wa_rstd(const T* src, int D, int dim, float eps, int lane) {
  float ss = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float f = ld_elem(src + d);
    ss += f * f;
  }
  return 1.f / sqrtf(warp_sum_f32(ss) / static_cast<float>(dim) + eps);
}

template <typename T>
__global__ void __launch_bounds__(128) qk_norm_append_kernel(WindowAttnParams p, int rows) {
  pdl_wait();
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const int heads = p.hq + 2 * p.hkv;
  if (warp >= rows * heads) return;
  const int row = warp / heads, head = warp % heads;
  T* base = static_cast<T*>(p.proj) + static_cast<size_t>(row) * p.stride;
  if (head < p.hq) {
    T* q = base + p.q_off + static_cast<size_t>(head) * p.D;
    const float r = wa_rstd(q, p.D, p.dim, p.eps, lane);
    for (int d = lane; d < p.D; d += 32) st_elem(q + d, ld_elem(q + d) * r * p.wq[d]);
    return;
  }
  const int32_t* bt = p.block_table + static_cast<size_t>(p.row_req[row]) * p.max_blocks;
  const int g = (head - p.hq) % p.hkv;
  const size_t tok = wa_token(p, bt, g, p.positions[row]);
  if (head < p.hq + p.hkv) {
    const T* k = base + p.k_off + static_cast<size_t>(g) * p.D;
    T* dst = static_cast<T*>(p.k_cache) + tok * p.D;
    const float r = wa_rstd(k, p.D, p.dim, p.eps, lane);
    for (int d = lane; d < p.D; d += 32) st_elem(dst + d, ld_elem(k + d) * r * p.wk[d]);
  } else {
    const T* v = base + p.v_off + static_cast<size_t>(g) * p.DV;
    T* dst = static_cast<T*>(p.v_cache) + tok * p.DV;
    for (int d = lane; d < p.DV; d += 32) dst[d] = v[d];
  }
}

// grid (hkv * head_chunks, splits, rows).  NG query heads of one kv head per CTA; a warp scores 32 keys at a time (lane =
// key), then the lanes take value columns 2 * lane + 64 * j.
template <typename T, int NV, int NG>
__global__ void __launch_bounds__(kWaWarps * 32) window_attn_kernel(WindowAttnParams p) {
  constexpr int DV = NV * 64, VN = Vec16<T>::N;
  extern __shared__ __align__(16) float wa_smem[];
  float* q_s = wa_smem;                                   // [NG][D]
  float* red_acc = q_s + NG * p.D;                        // [warps][NG][DV]
  __shared__ float red_m[kWaWarps][NG], red_l[kWaWarps][NG];
  pdl_wait();
  const int group = p.hq / p.hkv, chunks = (group + NG - 1) / NG;
  const int kvh = blockIdx.x / chunks, g0 = (blockIdx.x % chunks) * NG;
  const int split = blockIdx.y, row = p.row_list ? p.row_list[blockIdx.z] : static_cast<int>(blockIdx.z);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[row];
  const int ng = min(NG, group - g0), h0 = kvh * group + g0;
  const int first = max(0, pos + 1 - p.window), len = pos + 1;
  int per = (len - first + p.splits - 1) / p.splits;
  per = (per + 31) & ~31;
  const int t_begin = first + split * per;
  const int t_end = min(len, t_begin + per);
  const int32_t* bt = p.block_table + static_cast<size_t>(p.row_req[row]) * p.max_blocks;
  T* base = static_cast<T*>(p.proj) + static_cast<size_t>(row) * p.stride;
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);

  for (int g = warp; g < NG; g += kWaWarps) {
    const T* q = base + p.q_off + static_cast<size_t>(h0 + min(g, ng - 1)) * p.D;
    const float r = p.fused ? wa_rstd(q, p.D, p.dim, p.eps, lane) * p.scale : p.scale;
    for (int d = lane; d < p.D; d += 32) q_s[g * p.D + d] = ld_elem(q + d) * r * (p.fused ? p.wq[d] : 1.f);
  }
  if (p.fused && t_begin < len && t_end == len && warp == kWaWarps - 1) {
    // the CTA that reads the row's own position appends it (head chunks of one kv head write the same bytes)
    const size_t tok = wa_token(p, bt, kvh, pos);
    const T* k = base + p.k_off + static_cast<size_t>(kvh) * p.D;
    const T* v = base + p.v_off + static_cast<size_t>(kvh) * p.DV;
    const float r = wa_rstd(k, p.D, p.dim, p.eps, lane);
    T* kd = static_cast<T*>(p.k_cache) + tok * p.D;
    T* vd = static_cast<T*>(p.v_cache) + tok * p.DV;
    for (int d = lane; d < p.D; d += 32) st_elem(kd + d, ld_elem(k + d) * r * p.wk[d]);
    for (int d = lane; d < p.DV; d += 32) vd[d] = v[d];
  }
  __syncthreads();

  float m[NG], l[NG], acc[NG][2 * NV];
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    m[g] = -INFINITY;
    l[g] = 0.f;
#pragma unroll
    for (int j = 0; j < 2 * NV; ++j) acc[g][j] = 0.f;
  }
  for (int t0 = t_begin + warp * 32; t0 < t_end; t0 += kWaWarps * 32) {
    const int t = t0 + lane;
    const bool valid = t < t_end;
    const size_t tok = wa_token(p, bt, kvh, valid ? t : t_end - 1);
    float s[NG];
#pragma unroll
    for (int g = 0; g < NG; ++g) s[g] = 0.f;
    const T* kr = kc + tok * p.D;
#pragma unroll 4
    for (int c = 0; c < p.D; c += VN) {
      float kf[VN];
      Vec16<T>::load(kr + c, kf);
#pragma unroll
      for (int g = 0; g < NG; ++g) {
#pragma unroll
        for (int j = 0; j < VN; j += 4) {
          const float4 q4 = *reinterpret_cast<const float4*>(q_s + g * p.D + c + j);
          s[g] = fmaf(kf[j], q4.x, s[g]);
          s[g] = fmaf(kf[j + 1], q4.y, s[g]);
          s[g] = fmaf(kf[j + 2], q4.z, s[g]);
          s[g] = fmaf(kf[j + 3], q4.w, s[g]);
        }
      }
    }
    float pr[NG];
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      float tm = valid ? s[g] : -INFINITY;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, o));
      const float mn = fmaxf(m[g], tm);
      const float corr = m[g] == -INFINITY ? 0.f : wa_exp<T>(m[g] - mn);
      pr[g] = valid ? wa_exp<T>(s[g] - mn) : 0.f;
      l[g] = l[g] * corr + warp_sum_f32(pr[g]);
      m[g] = mn;
#pragma unroll
      for (int j = 0; j < 2 * NV; ++j) acc[g][j] *= corr;
    }
    const int n = min(32, t_end - t0);
    for (int tt = 0; tt < n; ++tt) {
      const size_t vtok = __shfl_sync(0xffffffffu, static_cast<unsigned long long>(tok), tt);
      const T* vr = vc + vtok * DV + 2 * lane;
      float2 vf[NV];
#pragma unroll
      for (int j = 0; j < NV; ++j) vf[j] = ld_elem2(vr + 64 * j);
#pragma unroll
      for (int g = 0; g < NG; ++g) {
        const float pg = __shfl_sync(0xffffffffu, pr[g], tt);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          acc[g][2 * j] = fmaf(pg, vf[j].x, acc[g][2 * j]);
          acc[g][2 * j + 1] = fmaf(pg, vf[j].y, acc[g][2 * j + 1]);
        }
      }
    }
  }
  if (lane == 0) {
#pragma unroll
    for (int g = 0; g < NG; ++g) { red_m[warp][g] = m[g]; red_l[warp][g] = l[g]; }
  }
#pragma unroll
  for (int g = 0; g < NG; ++g)
#pragma unroll
    for (int j = 0; j < NV; ++j)
      *reinterpret_cast<float2*>(red_acc + (warp * NG + g) * DV + 64 * j + 2 * lane) = make_float2(acc[g][2 * j], acc[g][2 * j + 1]);
  __syncthreads();
  for (int i = threadIdx.x; i < ng * DV; i += blockDim.x) {
    const int g = i / DV, d = i % DV;
    float mm = -INFINITY;
    for (int w = 0; w < kWaWarps; ++w) mm = fmaxf(mm, red_m[w][g]);
    float ll = 0.f, a = 0.f;
    for (int w = 0; w < kWaWarps; ++w) {
      const float c = red_m[w][g] == -INFINITY ? 0.f : wa_exp<T>(red_m[w][g] - mm);
      ll += red_l[w][g] * c;
      a += red_acc[(w * NG + g) * DV + d] * c;
    }
    const int h = h0 + g;
    if (p.splits == 1) {
      st_elem(static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_stride + static_cast<size_t>(h) * DV + d,
              ll > 0.f ? a / ll * p.out_scale : 0.f);
    } else {
      const size_t pi = (static_cast<size_t>(row) * p.hq + h) * p.splits + split;
      p.part_acc[pi * DV + d] = a;
      if (d == 0) { p.part_ml[pi * 2] = mm; p.part_ml[pi * 2 + 1] = ll; }
    }
  }
}

// grid (hq, rows), DV threads
template <typename T>
__global__ void __launch_bounds__(256) window_attn_combine_kernel(WindowAttnParams p) {
  pdl_wait();
  const int row = p.row_list ? p.row_list[blockIdx.y] : static_cast<int>(blockIdx.y);
  const int h = blockIdx.x, d = threadIdx.x;
  const size_t rh = static_cast<size_t>(row) * p.hq + h;
  float mm = -INFINITY;
  for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.part_ml[(rh * p.splits + s) * 2]);
  float ll = 0.f, a = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float ms = p.part_ml[(rh * p.splits + s) * 2];
    const float c = ms == -INFINITY ? 0.f : wa_exp<T>(ms - mm);
    ll += p.part_ml[(rh * p.splits + s) * 2 + 1] * c;
    a += p.part_acc[(rh * p.splits + s) * p.DV + d] * c;
  }
  st_elem(static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_stride + static_cast<size_t>(h) * p.DV + d,
          ll > 0.f ? a / ll * p.out_scale : 0.f);
}

template <typename T, int NV, int NG>
static int launch_wa(const WindowAttnParams& p, int rows, cudaStream_t st) {
  const int chunks = dgpp_ceil_div(p.hq / p.hkv, NG);
  const size_t smem = (static_cast<size_t>(NG) * p.D + static_cast<size_t>(kWaWarps) * NG * NV * 64) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(window_attn_kernel<T, NV, NG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    attr = true;
  }
  window_attn_kernel<T, NV, NG><<<dim3(p.hkv * chunks, p.splits, rows), kWaWarps * 32, smem, st>>>(p);
  DGPP_CUDA_OK(cudaGetLastError());
  if (p.splits > 1) {
    window_attn_combine_kernel<T><<<dim3(p.hq, rows), NV * 64, 0, st>>>(p);
    DGPP_CUDA_OK(cudaGetLastError());
  }
  return 0;
}

template <typename T, int NV>
static int launch_wa_g(const WindowAttnParams& p, int rows, cudaStream_t st) {
  const int g = p.hq / p.hkv;
  if (g == 1) return launch_wa<T, NV, 1>(p, rows, st);
  if (g == 2) return launch_wa<T, NV, 2>(p, rows, st);
  if (g <= 4) return launch_wa<T, NV, 4>(p, rows, st);
  return launch_wa<T, NV, 8>(p, rows, st);
}

template <typename T>
static int launch_wa_v(const WindowAttnParams& p, int rows, cudaStream_t st) {
  if (p.DV == 64) return launch_wa_g<T, 1>(p, rows, st);
  if (p.DV == 128) return launch_wa_g<T, 2>(p, rows, st);
  if (p.DV == 192) return launch_wa_g<T, 3>(p, rows, st);
  return launch_wa_g<T, 4>(p, rows, st);
}

static int wa_check(const WindowAttnParams& p, int rows) {
  DGPP_REQUIRE(p.hkv > 0 && p.hq % p.hkv == 0, "window_attn: %d query heads over %d key heads", p.hq, p.hkv);
  DGPP_REQUIRE(p.D % 64 == 0 && p.D >= 64 && p.D <= 256 && p.DV % 64 == 0 && p.DV >= 64 && p.DV <= 256,
               "window_attn: head widths %d / %d (padded to multiples of 64, at most 256)", p.D, p.DV);
  DGPP_REQUIRE(p.stride % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 && p.v_off % 8 == 0, "window_attn: unaligned projection rows");
  DGPP_REQUIRE(p.window >= 1 && p.splits >= 1 && p.page >= 1 && p.dim >= 1 && p.dim <= p.D, "window_attn: window %d splits %d", p.window, p.splits);
  DGPP_REQUIRE(p.splits == 1 || (p.part_ml && p.part_acc), "window_attn: scratch required when splits > 1");
  DGPP_REQUIRE(rows >= 0 && rows <= 65535, "window_attn: %d rows", rows);
  return 0;
}

}  // namespace dgpp

using namespace dgpp;

static WindowAttnParams wa_params(void* proj, int64_t stride, int q_off, int k_off, int v_off, const void* wq, const void* wk,
                                  void* k_cache, void* v_cache, const void* block_table, const void* row_req,
                                  const void* positions, int hq, int hkv, int D, int DV, int dim, int page, int max_blocks, float eps) {
  WindowAttnParams p;
  p.proj = proj; p.stride = stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  p.wq = static_cast<const float*>(wq); p.wk = static_cast<const float*>(wk);
  p.k_cache = k_cache; p.v_cache = v_cache;
  p.block_table = static_cast<const int32_t*>(block_table);
  p.row_req = static_cast<const int32_t*>(row_req);
  p.positions = static_cast<const int32_t*>(positions);
  p.row_list = nullptr; p.part_ml = nullptr; p.part_acc = nullptr; p.out = nullptr; p.out_stride = 0;
  p.hq = hq; p.hkv = hkv; p.D = D; p.DV = DV; p.dim = dim; p.page = page; p.max_blocks = max_blocks;
  p.splits = 1; p.window = 1; p.fused = 0; p.scale = 1.f; p.eps = eps; p.out_scale = 1.f;
  return p;
}

DGPP_API int dgpp_qk_norm_append(void* proj, int64_t stride, int q_off, int k_off, int v_off, const void* wq, const void* wk,
                                 void* k_cache, void* v_cache, const void* block_table, const void* row_req, const void* positions,
                                 int rows, int hq, int hkv, int D, int DV, int dim, int page, int max_blocks, float eps, int f32,
                                 cudaStream_t st) {
  const WindowAttnParams p = wa_params(proj, stride, q_off, k_off, v_off, wq, wk, k_cache, v_cache, block_table, row_req, positions,
                                       hq, hkv, D, DV, dim, page, max_blocks, eps);
  if (wa_check(p, rows)) return -1;
  if (rows == 0) return 0;
  const int blocks = dgpp_ceil_div(rows * (hq + 2 * hkv), 4);
  if (f32) qk_norm_append_kernel<float><<<blocks, 128, 0, st>>>(p, rows);
  else qk_norm_append_kernel<bf16><<<blocks, 128, 0, st>>>(p, rows);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// rows: rows of this launch (row_list, int32, names them when given).  fused: see the header.  out_scale multiplies the
// outputs before they are rounded.  part_ml / part_acc: rows of the whole pass * hq * splits * (2 | DV) floats.
DGPP_API int dgpp_window_attn(void* proj, int64_t stride, int q_off, int k_off, int v_off, const void* wq, const void* wk,
                              void* k_cache, void* v_cache, const void* block_table, const void* row_req, const void* positions,
                              const void* row_list, void* part_ml, void* part_acc, void* out, int64_t out_stride, int rows,
                              int hq, int hkv, int D, int DV, int dim, int page, int max_blocks, int splits, int window, int fused,
                              float scale, float eps, float out_scale, int f32, cudaStream_t st) {
  WindowAttnParams p = wa_params(proj, stride, q_off, k_off, v_off, wq, wk, k_cache, v_cache, block_table, row_req, positions,
                                 hq, hkv, D, DV, dim, page, max_blocks, eps);
  p.row_list = static_cast<const int32_t*>(row_list);
  p.part_ml = static_cast<float*>(part_ml); p.part_acc = static_cast<float*>(part_acc);
  p.out = out; p.out_stride = out_stride;
  p.splits = splits; p.window = window; p.fused = fused; p.scale = scale; p.out_scale = out_scale;
  if (wa_check(p, rows)) return -1;
  if (rows == 0) return 0;
  return f32 ? launch_wa_v<float>(p, rows, st) : launch_wa_v<bf16>(p, rows, st);
}

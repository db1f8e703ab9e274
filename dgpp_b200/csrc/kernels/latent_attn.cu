// Sliding-window latent attention for 16-bit and true 32-bit activations: what lies around the tensor-core kernels
// (mla_tc.cu for single tokens, window_attn_tc.cu for prompt runs), and a CUDA-core attention kernel for the rest.
//
// A cache row holds [latent c (KC columns) | rotated key part (RP columns)], shared by every head.  Per head the key is
// [W_uk c | rotated part] and the value W_uv c; the up matrices sit in one matrix w_up [heads * DN + heads * DV, KC], key rows first.
//
//   latent_append   prompt rows: RMS norm of c, rotation of the shared key part, both into the paged cache; rotates the queries in
//                   place (neighbouring pairs, the first `rot` columns of the rotated part)
//   latent_absorb   q_abs[row, head] = [W_uk^T q_plain | q_rotated] in fp32; fused: rows are new tokens, the kernel rotates their
//                   queries itself and appends their cache rows (one launch in front of the attention of a decode pass)
//   latent_rows     attention of single rows on the CUDA cores, any widths: scores q_abs . cache row, output sum p c (fp32)
//   latent_up       out[row, head] = W_uv lat[row, head] * sigmoid(gate[row, head])
//   latent_gather   pages of the cache into consecutive rows (the input of the up-projection that expands a prompt's keys)
//
// Angles: common/rope.cuh.
#include <math.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"
#include "common/rope.cuh"

namespace dgpp {

struct LatentArgs {
  void* proj;               // [rows, stride] (T): queries [heads, DN + RP] from q_off, [c | key part] from kv_off
  int64_t stride;
  int q_off, kv_off;
  const float* norm_w;      // [rank]
  const float* freq;        // [2, rot / 2]: rotation frequencies, leading and residual term
  const int32_t* positions;
  const int32_t* row_req;
  const int32_t* block_table;
  const int32_t* row_list;  // optional: pass rows of this launch
  void* cache;              // [blocks, page, KC + RP] (T)
  const void* w_up;         // [heads * (DN + DV), KC] (T)
  float* q_abs;             // [n, heads, KC + RP]
  int n, heads, DN, DV, dim, rank, KC, RP, rot_dim, rot, page, max_blocks, fused;
  float eps;
};

// One warp: the cache row of one token.
template <typename T>
__device__ __forceinline__ void latent_cache_row(const LatentArgs& a, int row, int lane) {
  const T* src = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.kv_off;
  const int pos = a.positions[row];
  const int blk = a.block_table[static_cast<size_t>(a.row_req[row]) * a.max_blocks + pos / a.page];
  T* dst = static_cast<T*>(a.cache) + (static_cast<size_t>(blk) * a.page + pos % a.page) * (a.KC + a.RP);
  float ss = 0.f;
  for (int i = lane; i < a.rank; i += 32) {
    const float v = ld_elem(src + i);
    ss = fmaf(v, v, ss);
  }
  const float r = 1.f / sqrtf(warp_sum_f32(ss) / static_cast<float>(a.rank) + a.eps);
  for (int i = lane; i < a.KC; i += 32) st_elem(dst + i, i < a.rank ? ld_elem(src + i) * r * a.norm_w[i] : 0.f);
  const T* kr = src + a.KC;
  for (int i = lane; i < a.RP / 2; i += 32) {
    float u = ld_elem(kr + 2 * i), v = ld_elem(kr + 2 * i + 1);
    if (2 * i < a.rot) {
      float s, c;
      rope_angle(a.freq, a.rot / 2, pos, i, s, c);
      const float t = u * c - v * s;
      v = v * c + u * s;
      u = t;
    }
    st_elem(dst + a.KC + 2 * i, u);
    st_elem(dst + a.KC + 2 * i + 1, v);
  }
}

// grid (rows), 256 threads
template <typename T>
__global__ void __launch_bounds__(256) latent_append_kernel(LatentArgs a) {
  extern __shared__ float la_cs[];                        // [rot / 2][2]
  pdl_wait();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < a.rot / 2; i += 256) rope_angle(a.freq, a.rot / 2, a.positions[row], i, la_cs[2 * i], la_cs[2 * i + 1]);
  __syncthreads();
  if (warp == 0) latent_cache_row<T>(a, row, lane);
  T* q = static_cast<T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.q_off;
  for (int h = warp; h < a.heads; h += 8) {
    T* qr = q + static_cast<size_t>(h) * (a.DN + a.RP) + a.DN;
    for (int i = lane; i < a.rot / 2; i += 32) {
      const float u = ld_elem(qr + 2 * i), v = ld_elem(qr + 2 * i + 1), s = la_cs[2 * i], c = la_cs[2 * i + 1];
      st_elem(qr + 2 * i, u * c - v * s);
      st_elem(qr + 2 * i + 1, v * c + u * s);
    }
  }
}

constexpr int kLatRows = 8;

// grid (heads (+ 1 when fused), ceil(n / 8), KC / 128 rounded up), 256 threads: a CTA owns 128 latent columns of one head for up to
// 8 rows; a warp sums an eighth of the head's key rows (lane = four columns), the eight partial sums are added in warp order.  The
// CTAs behind the last head write the cache rows.
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(LatentArgs a) {
  extern __shared__ __align__(16) float ab_smem[];
  float* qs = ab_smem;                                    // [dim][8 rows]
  float* part = ab_smem + kLatRows * a.dim;               // [8 warps][8 rows][128]
  pdl_wait();
  const int h = blockIdx.x, r0 = blockIdx.y * kLatRows, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nr = min(kLatRows, a.n - r0);
  auto pass_row = [&](int r) { return a.row_list != nullptr ? a.row_list[r0 + r] : r0 + r; };
  if (h == a.heads) {
    if (blockIdx.z == 0 && warp < nr) latent_cache_row<T>(a, pass_row(warp), lane);
    return;
  }
  const T* proj = static_cast<const T*>(a.proj);
  const size_t qcol = a.q_off + static_cast<size_t>(h) * (a.DN + a.RP);
  if (warp < kLatRows) {
    const T* src = proj + static_cast<size_t>(pass_row(min(warp, nr - 1))) * a.stride + qcol;
    for (int c = lane; c < a.dim; c += 32) qs[c * kLatRows + warp] = warp < nr ? ld_elem(src + c) : 0.f;
  }
  __syncthreads();
  const int d0 = blockIdx.z * 128 + lane * 4;
  const bool live = d0 < a.KC;
  const int per = (a.dim + 7) / 8, n0 = warp * per, n1 = live ? min(a.dim, n0 + per) : n0;
  float acc[kLatRows][4];
#pragma unroll
  for (int r = 0; r < kLatRows; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
  const T* wp = static_cast<const T*>(a.w_up) + static_cast<size_t>(h) * a.DN * a.KC + (live ? d0 : 0);
#pragma unroll 8
  for (int c = n0; c < n1; ++c) {
    const float4 w = ld_elem4(wp + static_cast<size_t>(c) * a.KC);
    const float4 qa = *reinterpret_cast<const float4*>(qs + c * kLatRows), qb = *reinterpret_cast<const float4*>(qs + c * kLatRows + 4);
    const float q[kLatRows] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
    for (int r = 0; r < kLatRows; ++r) {
      acc[r][0] = fmaf(q[r], w.x, acc[r][0]);
      acc[r][1] = fmaf(q[r], w.y, acc[r][1]);
      acc[r][2] = fmaf(q[r], w.z, acc[r][2]);
      acc[r][3] = fmaf(q[r], w.w, acc[r][3]);
    }
  }
#pragma unroll
  for (int r = 0; r < kLatRows; ++r)
    *reinterpret_cast<float4*>(part + (warp * kLatRows + r) * 128 + lane * 4) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
  __syncthreads();
  const int D = a.KC + a.RP;
  {
    const int r = warp, d = lane * 4;                     // 8 warps = 8 rows
    if (r < nr && live) {
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float4 v = *reinterpret_cast<const float4*>(part + (w * kLatRows + r) * 128 + d);
        sum.x += v.x; sum.y += v.y; sum.z += v.z; sum.w += v.w;
      }
      *reinterpret_cast<float4*>(a.q_abs + (static_cast<size_t>(r0 + r) * a.heads + h) * D + d0) = sum;
    }
  }
  if (blockIdx.z != 0) return;
  for (int i = tid; i < nr * (a.RP / 2); i += 256) {
    const int r = i / (a.RP / 2), j = i % (a.RP / 2), row = pass_row(r);
    const T* qr = proj + static_cast<size_t>(row) * a.stride + qcol + a.DN + 2 * j;
    float u = ld_elem(qr), v = ld_elem(qr + 1);
    if (a.fused && 2 * j < a.rot) {
      float s, c;
      rope_angle(a.freq, a.rot / 2, a.positions[row], j, s, c);
      const float t = u * c - v * s;
      v = v * c + u * s;
      u = t;
    }
    float* o = a.q_abs + (static_cast<size_t>(r0 + r) * a.heads + h) * D + a.KC + 2 * j;
    o[0] = u;
    o[1] = v;
  }
}

struct LatentRowsArgs {
  const float* q;           // [n, heads, KC + RP]
  const void* cache;
  const int32_t* block_table;
  const int32_t* row_req;
  const int32_t* positions;
  const int32_t* row_list;
  float* out;               // [n, heads, KC]
  int n, heads, KC, RP, page, max_blocks, window;
  float scale;
};

constexpr int kLrTile = 32, kLrHeads = 8;

// grid (n, ceil(heads / 8)), 256 threads: a warp is one head; 32 cache rows at a time in shared memory (odd stride in words), lane =
// token for the scores, lane = columns lane + 32 j of the output.
template <typename T, int PER>
__global__ void __launch_bounds__(256) latent_rows_kernel(LatentRowsArgs a) {
  extern __shared__ __align__(16) float lr_smem[];
  const int D = a.KC + a.RP, DS = D + static_cast<int>(4 / sizeof(T));       // shared row stride: D words are even, one more is odd
  float* qs = lr_smem;                                     // [8][D]
  T* tile = reinterpret_cast<T*>(qs + kLrHeads * D);       // [32][DS]
  pdl_wait();
  const int i0 = blockIdx.x, row = a.row_list != nullptr ? a.row_list[i0] : i0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y * kLrHeads + warp;
  const int pos = a.positions[row], first = max(0, pos + 1 - a.window), len = pos + 1;
  const int32_t* bt = a.block_table + static_cast<size_t>(a.row_req[row]) * a.max_blocks;
  for (int i = tid; i < kLrHeads * D; i += 256) {
    const int hh = min(static_cast<int>(blockIdx.y) * kLrHeads + i / D, a.heads - 1);
    qs[i] = a.q[(static_cast<size_t>(i0) * a.heads + hh) * D + i % D] * a.scale;
  }
  float m = -INFINITY, l = 0.f, acc[PER];
#pragma unroll
  for (int j = 0; j < PER; ++j) acc[j] = 0.f;
  for (int t0 = first; t0 < len; t0 += kLrTile) {
    const int n = min(kLrTile, len - t0);
    __syncthreads();
    for (int i = tid; i < kLrTile * (D / 2); i += 256) {
      const int t = i / (D / 2), c = (i % (D / 2)) * 2;
      float2 v = make_float2(0.f, 0.f);
      if (t < n) v = ld_elem2(static_cast<const T*>(a.cache) + (static_cast<size_t>(bt[(t0 + t) / a.page]) * a.page + (t0 + t) % a.page) * D + c);
      st_elem(tile + t * DS + c, v.x);
      st_elem(tile + t * DS + c + 1, v.y);
    }
    __syncthreads();
    const T* tr = tile + lane * DS;
    const float* q = qs + warp * D;
    float s = 0.f;
#pragma unroll 4
    for (int c = 0; c < D; ++c) s = fmaf(ld_elem(tr + c), q[c], s);
    float tm = lane < n ? s : -INFINITY;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, o));
    const float mn = fmaxf(m, tm), corr = m == -INFINITY ? 0.f : expf(m - mn);
    const float p = lane < n ? expf(s - mn) : 0.f;
    l = l * corr + warp_sum_f32(p);
    m = mn;
#pragma unroll
    for (int j = 0; j < PER; ++j) acc[j] *= corr;
    for (int t = 0; t < n; ++t) {
      const float pt = __shfl_sync(0xffffffffu, p, t);
#pragma unroll
      for (int j = 0; j < PER; ++j)
        if (lane + 32 * j < a.KC) acc[j] = fmaf(pt, ld_elem(tile + t * DS + lane + 32 * j), acc[j]);
    }
  }
  if (h >= a.heads) return;
#pragma unroll
  for (int j = 0; j < PER; ++j)
    if (lane + 32 * j < a.KC) a.out[(static_cast<size_t>(i0) * a.heads + h) * a.KC + lane + 32 * j] = acc[j] / l;
}

constexpr int kUpOut = 4;        // outputs of a lane

// grid (heads, ceil(n / 8), ceil(DV / 64)), 256 threads: a CTA owns 64 outputs of one head for up to 8 rows.  Sixteen lanes take the
// 16-byte chunks of four weight rows in turns, so a value read from shared memory meets four weights.
template <typename T>
__global__ void __launch_bounds__(256) latent_up_kernel(const float* __restrict__ lat, const T* __restrict__ w, const T* __restrict__ gate,
                                                        int64_t gate_stride, const int32_t* __restrict__ row_list, T* __restrict__ out,
                                                        int64_t out_stride, int n, int heads, int DV, int KC) {
  constexpr int VN = Vec16<T>::N, CS = VN + 4;             // a chunk of VN values takes CS words: 16-byte reads without bank conflicts
  extern __shared__ __align__(16) float lu_smem[];         // [8][chunks][CS]
  pdl_wait();
  const int h = blockIdx.x, r0 = blockIdx.y * kLatRows, tid = threadIdx.x, nr = min(kLatRows, n - r0), chunks = KC / VN;
  const int warp = tid >> 5, lane = tid & 31, g = lane & 15;
  {
    const int r = warp;                                    // 8 warps = 8 rows
    const float* src = lat + (static_cast<size_t>(r0 + min(r, nr - 1)) * heads + h) * KC;
    for (int d = lane * 4; d < KC; d += 128)
      *reinterpret_cast<float4*>(lu_smem + (r * chunks + d / VN) * CS + d % VN) = r < nr ? *reinterpret_cast<const float4*>(src + d) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  __syncthreads();
  const int v0 = blockIdx.z * 64 + (warp * 2 + (lane >> 4)) * kUpOut;
  const T* wp = w + static_cast<size_t>(h) * DV * KC;
  float acc[kUpOut][kLatRows];
#pragma unroll
  for (int o = 0; o < kUpOut; ++o)
#pragma unroll
    for (int r = 0; r < kLatRows; ++r) acc[o][r] = 0.f;
  for (int c = g; c < chunks; c += 16) {
    float f[kUpOut][VN];
#pragma unroll
    for (int o = 0; o < kUpOut; ++o) Vec16<T>::load(wp + static_cast<size_t>(min(v0 + o, DV - 1)) * KC + c * VN, f[o]);
#pragma unroll
    for (int r = 0; r < kLatRows; ++r) {
#pragma unroll
      for (int j = 0; j < VN; j += 4) {
        const float4 x = *reinterpret_cast<const float4*>(lu_smem + (r * chunks + c) * CS + j);
#pragma unroll
        for (int o = 0; o < kUpOut; ++o)
          acc[o][r] = fmaf(x.w, f[o][j + 3], fmaf(x.z, f[o][j + 2], fmaf(x.y, f[o][j + 1], fmaf(x.x, f[o][j], acc[o][r]))));
      }
    }
  }
#pragma unroll
  for (int o = 0; o < kUpOut; ++o)
#pragma unroll
    for (int r = 0; r < kLatRows; ++r) {
      float s = acc[o][r];
#pragma unroll
      for (int k = 8; k > 0; k >>= 1) s += __shfl_xor_sync(0xffffffffu, s, k);
      if (g == r && v0 + o < DV && r < nr) {               // lane r of the sixteen finishes row r
        const size_t row = row_list != nullptr ? row_list[r0 + r] : r0 + r;
        st_elem(out + row * out_stride + static_cast<size_t>(h) * DV + v0 + o, s * sigmoid_f32(ld_elem(gate + row * gate_stride + h)));
      }
    }
}

// grid (pages), 256 threads
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, const int32_t* __restrict__ pages, uint4* __restrict__ out,
                                                            int vecs) {
  pdl_wait();
  const uint4* src = cache + static_cast<size_t>(pages[blockIdx.x]) * vecs;
  uint4* dst = out + static_cast<size_t>(blockIdx.x) * vecs;
  for (int i = threadIdx.x; i < vecs; i += 256) dst[i] = src[i];
}

static int latent_check(const LatentArgs& a) {
  DGPP_REQUIRE(a.KC % 64 == 0 && a.KC >= 64 && a.rank >= 1 && a.rank <= a.KC && a.RP % 64 == 0 && a.rot_dim <= a.RP && a.rot >= 0 &&
                   a.rot % 2 == 0 && a.rot <= a.rot_dim, "latent: rank %d of %d, rotated part %d (%d turned) of %d", a.rank, a.KC, a.rot_dim, a.rot, a.RP);
  DGPP_REQUIRE(a.dim >= 1 && a.dim <= a.DN && a.heads >= 1 && a.n >= 0 && a.n <= 65535 * kLatRows, "latent: %d heads of %d in %d columns", a.heads, a.dim, a.DN);
  return 0;
}

}  // namespace dgpp

using namespace dgpp;

static LatentArgs latent_args(void* proj, int64_t stride, int q_off, int kv_off, const void* norm_w, const void* freq, const void* positions,
                              const void* row_req, const void* block_table, void* cache, int n, int heads, int DN, int DV, int dim, int rank, int KC,
                              int RP, int rot_dim, int rot, int page, int max_blocks, float eps) {
  LatentArgs a = {};
  a.proj = proj; a.stride = stride; a.q_off = q_off; a.kv_off = kv_off;
  a.norm_w = static_cast<const float*>(norm_w); a.freq = static_cast<const float*>(freq);
  a.positions = static_cast<const int32_t*>(positions); a.row_req = static_cast<const int32_t*>(row_req);
  a.block_table = static_cast<const int32_t*>(block_table);
  a.cache = cache;
  a.n = n; a.heads = heads; a.DN = DN; a.DV = DV; a.dim = dim; a.rank = rank; a.KC = KC; a.RP = RP; a.rot_dim = rot_dim; a.rot = rot;
  a.page = page; a.max_blocks = max_blocks; a.eps = eps;
  return a;
}

DGPP_API int dgpp_latent_append(void* proj, int64_t stride, int q_off, int kv_off, const void* norm_w, const void* freq, const void* positions,
                                const void* row_req, const void* block_table, void* cache, int rows, int heads, int DN, int DV, int dim, int rank,
                                int KC, int RP, int rot_dim, int rot, int page, int max_blocks, float eps, int f32, cudaStream_t st) {
  const LatentArgs a = latent_args(proj, stride, q_off, kv_off, norm_w, freq, positions, row_req, block_table, cache, rows, heads, DN, DV, dim,
                                   rank, KC, RP, rot_dim, rot, page, max_blocks, eps);
  if (latent_check(a)) return -1;
  if (rows == 0) return 0;
  const size_t smem = static_cast<size_t>(rot) * sizeof(float);
  if (f32) latent_append_kernel<float><<<rows, 256, smem, st>>>(a);
  else latent_append_kernel<bf16><<<rows, 256, smem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// n rows (row_list names their pass rows when given).  fused: see the header; else latent_append has run.
DGPP_API int dgpp_latent_absorb(void* proj, int64_t stride, int q_off, int kv_off, const void* norm_w, const void* freq, const void* positions,
                                const void* row_req, const void* block_table, void* cache, const void* row_list, const void* w_up, void* q_abs,
                                int n, int heads, int DN, int DV, int dim, int rank, int KC, int RP, int rot_dim, int rot, int page, int max_blocks,
                                int fused, float eps, int f32, cudaStream_t st) {
  LatentArgs a = latent_args(proj, stride, q_off, kv_off, norm_w, freq, positions, row_req, block_table, cache, n, heads, DN, DV, dim, rank, KC,
                             RP, rot_dim, rot, page, max_blocks, eps);
  if (latent_check(a)) return -1;
  DGPP_REQUIRE(dim <= 1024, "latent_absorb: heads of %d columns (at most 1024)", dim);
  if (n == 0) return 0;
  a.row_list = static_cast<const int32_t*>(row_list); a.w_up = w_up; a.q_abs = static_cast<float*>(q_abs); a.fused = fused;
  const dim3 grid(heads + (fused ? 1 : 0), dgpp_ceil_div(n, kLatRows), dgpp_ceil_div(KC, 128));
  const size_t smem = static_cast<size_t>(kLatRows * dim + 8 * kLatRows * 128) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(latent_absorb_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    DGPP_CUDA_OK(cudaFuncSetAttribute(latent_absorb_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    attr = true;
  }
  if (f32) latent_absorb_kernel<float><<<grid, 256, smem, st>>>(a);
  else latent_absorb_kernel<bf16><<<grid, 256, smem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename T, int PER>
static int launch_latent_rows(const LatentRowsArgs& a, cudaStream_t st) {
  const int D = a.KC + a.RP;
  const size_t smem = static_cast<size_t>(kLrHeads) * D * sizeof(float) + static_cast<size_t>(kLrTile) * (D + 4 / sizeof(T)) * sizeof(T);
  DGPP_REQUIRE(smem <= 227 * 1024, "latent_rows: cache rows of %d columns do not fit shared memory", D);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(latent_rows_kernel<T, PER>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    attr = true;
  }
  latent_rows_kernel<T, PER><<<dim3(a.n, dgpp_ceil_div(a.heads, kLrHeads)), 256, smem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename T>
static int launch_latent_rows_per(const LatentRowsArgs& a, cudaStream_t st) {
  if (a.KC <= 128) return launch_latent_rows<T, 4>(a, st);
  if (a.KC <= 512) return launch_latent_rows<T, 16>(a, st);
  return launch_latent_rows<T, 32>(a, st);
}

// Windowed attention of n rows on the CUDA cores -> out [n, heads, KC] fp32.
DGPP_API int dgpp_latent_rows(const void* q, const void* cache, const void* block_table, const void* row_req, const void* positions,
                              const void* row_list, void* out, int n, int heads, int KC, int RP, int page, int max_blocks, int window, float scale,
                              int f32, cudaStream_t st) {
  DGPP_REQUIRE(KC % 64 == 0 && KC >= 64 && KC <= 1024 && RP % 64 == 0 && window >= 1, "latent_rows: cache rows %d + %d, window %d", KC, RP, window);
  if (n == 0) return 0;
  LatentRowsArgs a = {};
  a.q = static_cast<const float*>(q); a.cache = cache;
  a.block_table = static_cast<const int32_t*>(block_table);
  a.row_req = static_cast<const int32_t*>(row_req); a.positions = static_cast<const int32_t*>(positions);
  a.row_list = static_cast<const int32_t*>(row_list); a.out = static_cast<float*>(out);
  a.n = n; a.heads = heads; a.KC = KC; a.RP = RP; a.page = page; a.max_blocks = max_blocks; a.window = window; a.scale = scale;
  return f32 ? launch_latent_rows_per<float>(a, st) : launch_latent_rows_per<bf16>(a, st);
}

// lat [n, heads, KC] fp32, w [heads * DV, KC], gate: one column per head (row stride gate_stride) -> columns h * DV + v of out.
DGPP_API int dgpp_latent_up(const void* lat, const void* w, const void* gate, int64_t gate_stride, const void* row_list, void* out,
                            int64_t out_stride, int n, int heads, int DV, int KC, int f32, cudaStream_t st) {
  DGPP_REQUIRE(KC % 64 == 0 && KC <= 1024 && DV >= 1, "latent_up: %d columns from %d", DV, KC);
  if (n == 0) return 0;
  const dim3 grid(heads, dgpp_ceil_div(n, kLatRows), dgpp_ceil_div(DV, 64));
  const int vn = f32 ? 4 : 8;
  const size_t smem = static_cast<size_t>(kLatRows) * (KC / vn) * (vn + 4) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(latent_up_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    DGPP_CUDA_OK(cudaFuncSetAttribute(latent_up_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    attr = true;
  }
  const float* lp = static_cast<const float*>(lat);
  const int32_t* rl = static_cast<const int32_t*>(row_list);
  if (f32) latent_up_kernel<float><<<grid, 256, smem, st>>>(lp, static_cast<const float*>(w), static_cast<const float*>(gate), gate_stride, rl, static_cast<float*>(out), out_stride, n, heads, DV, KC);
  else latent_up_kernel<bf16><<<grid, 256, smem, st>>>(lp, static_cast<const bf16*>(w), static_cast<const bf16*>(gate), gate_stride, rl, static_cast<bf16*>(out), out_stride, n, heads, DV, KC);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// pages [n] physical page ids; out [n * page, cols] (16-bit elements).
DGPP_API int dgpp_latent_gather(const void* cache, const void* pages, void* out, int n, int page, int cols, cudaStream_t st) {
  DGPP_REQUIRE(cols % 8 == 0, "latent_gather: rows of %d columns (a multiple of 8)", cols);
  if (n == 0) return 0;
  latent_gather_kernel<<<n, 256, 0, st>>>(static_cast<const uint4*>(cache), static_cast<const int32_t*>(pages), static_cast<uint4*>(out), page * cols / 8);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

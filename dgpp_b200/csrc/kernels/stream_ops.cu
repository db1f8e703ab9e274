// Row operators of models that keep the residual stream in fp32 (activations T = bf16 or fp32):
//   embed_rows        out[r] = scale * table[ids[r]]                           (fp32 rows; on request a second time in T)
//   resid_norm        x += delta (fp32, optional); out = x / sqrt(mean(x^2) + eps) * w           (out in T)
//   gated_group_norm  per group of columns: out = o / sqrt(mean(o^2) + eps) * w * act(gate) * scale; act: sigmoid or silu; o may first be
//                     divided by a number per row and group
//   geglu             out = gelu_tanh(gate) * up
//   stream_norm       x += mult * post(delta + bias) + vec; out = pre(x); post and pre each nothing, an RMS norm (over the row, or over
//                     each of several equal parts of it) or a layer norm (weight, perhaps a bias); delta is a row of fp32, or the sum of
//                     two such rows, each behind an RMS norm and a bias of its own, or the weighed rows of a mixture of experts (some of
//                     which may be the block's input itself) plus its shared expert, gated or not; vec is one row for all
//   gated_part_norm   a = y * silu(z); every one of `parts` runs of columns by its own root mean square, times w
//   clamped_glu       g = min(s gate, limit), u = clamp(s up, -limit, limit); out = r * g * sigmoid(alpha g) * (u + shift); s or r: a
//                     factor per row (the weight of a routed expert on its input or on its output; the products with the weights
//                     are linear), else one
//   act_rows          out = r * act(x); act: square of relu, or gelu (erf form); r: a factor per row, else one
//   token_gate        out = gelu_tanh(gate) * table[ids[r]][columns of one layer]
//   softcap           x = cap * tanh(x / cap)
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
embed_rows_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, T* __restrict__ copy, int64_t copy_stride,
                  int cols, int vocab, float scale) {
  pdl_wait();
  const int row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + static_cast<size_t>(id) * cols;
  float* dst = out + static_cast<size_t>(row) * cols;
  for (int i = threadIdx.x * 4; i < cols; i += kStreamThreads * 4) {
    float4 v = ld_elem4(src + i);
    v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
    st_elem4(dst + i, v);
    if (copy != nullptr) st_elem4(copy + row * copy_stride + i, v);
  }
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

// o [rows, groups * gp] fp32, gate [rows, gate_stride] (TG), w [gp] shared by the groups, or one row per group w_stride apart; den [rows,
// groups] or null.  A group is handled by `team` threads
// (a warp, or the whole CTA for wide groups).
template <typename T, typename TG>
__global__ void __launch_bounds__(kStreamThreads)
gated_group_norm_kernel(const float* __restrict__ o, const float* __restrict__ den, const TG* __restrict__ gate, int64_t gate_stride,
                        const float* __restrict__ w, int w_stride, T* __restrict__ out, int64_t out_stride, int rows, int groups, int gp, int n, float eps, float scale, int silu, int team) {
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
  const float inv = den != nullptr ? 1.f / den[row * groups + g] : 1.f;
  const float r = scale * inv / sqrtf(ss * inv * inv / static_cast<float>(n) + eps);
  w += static_cast<size_t>(g) * w_stride;
  for (int i = me * 4; i < gp; i += team * 4) {
    const float4 v = ld_elem4(op + i), a = ld_elem4(gt + i), ww = ld_elem4(w + i);
    auto act = [silu](float z) { return silu ? silu_f32(z) : sigmoid_f32(z); };
    st_elem4(dst + i, make_float4(v.x * r * ww.x * act(a.x), v.y * r * ww.y * act(a.y), v.z * r * ww.z * act(a.z), v.w * r * ww.w * act(a.w)));
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

enum NormKind { kNormNone = 0, kNormRms = 1, kNormLayer = 2, kNormParts = 3 };

// The rows of a mixture of experts that make up a delta: sum over j of y[pair_row[r * top + j]] (fp32, ascending j) and, with a
// shared expert, sigmoid(gate[r]) * shared[r] (no gate: shared[r]).  A negative pair_row is the block's input `self` itself, times
// its weight wts[r * top + j].
template <typename T>
struct MoeRows {
  const T* y;
  const int32_t* pair_row;
  const T* shared;
  const float* gate;
  int64_t gate_stride;
  const T* self;
  const float* wts;
  int top;
};

// A delta that is the sum of two rows: half (rms(delta + bias) * w + rms(second + second_b) * second_w) with half = factor.
struct SecondRow {
  const float *row, *bias, *w, *first_w;
  float factor;
};

struct RowNorm {
  int kind;
  const float *w, *b;        // weights; bias or null
};

// v += one row of fp32 (or nothing)
template <int NT, int NV>
__device__ __forceinline__ void add_row(float4 (&v)[NV], const float* __restrict__ b, int cols) {
  if (b == nullptr) return;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    if (i < cols) {
      const float4 e = ld_elem4(b + i);
      v[j].x += e.x; v[j].y += e.y; v[j].z += e.z; v[j].w += e.w;
    }
  }
}

// Norm of a row held in registers; columns at or beyond n are zero and stay zero (their weights and biases are zero).
template <int NT, int NV>
__device__ __forceinline__ void norm_row(float4 (&v)[NV], const RowNorm& norm, int cols, int n, float eps, float* scratch) {
  const int kind = norm.kind;
  if (kind == kNormNone) return;
  float mean = 0.f;
  if (kind == kNormLayer) {
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) sum += (v[j].x + v[j].y) + (v[j].z + v[j].w);
    mean = block_sum_f32(sum, scratch) / static_cast<float>(n);
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    float* f = reinterpret_cast<float*>(&v[j]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (kind == kNormLayer) f[e] = (threadIdx.x + NT * j) * 4 + e < n ? f[e] - mean : 0.f;
      ss = fmaf(f[e], f[e], ss);
    }
  }
  const float r = 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(n) + eps);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    if (i < cols) {
      const float4 g = ld_elem4(norm.w + i);
      v[j].x *= r * g.x; v[j].y *= r * g.y; v[j].z *= r * g.z; v[j].w *= r * g.w;
    }
  }
  add_row<NT, NV>(v, norm.b, cols);
}

// RMS norm of `parts` equal runs of a row's n true columns.  smem: cols + parts floats, shared by the calls of a kernel.
template <int NT, int NV>
__device__ __forceinline__ void norm_parts(float4 (&v)[NV], const RowNorm& norm, int cols, int n, int parts, float eps, float* smem) {
  const int len = n / parts, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool quad = len % 4 == 0;                          // four columns always belong to one part
  float* rs = smem + cols;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    if (i >= cols) continue;
    const float4 q = make_float4(v[j].x * v[j].x, v[j].y * v[j].y, v[j].z * v[j].z, v[j].w * v[j].w);
    if (quad) smem[i >> 2] = (q.x + q.y) + (q.z + q.w);
    else *reinterpret_cast<float4*>(smem + i) = q;
  }
  __syncthreads();
  const int entries = quad ? len >> 2 : len;
  for (int g = warp; g < parts; g += NT / 32) {
    float ss = 0.f;
    for (int k = lane; k < entries; k += 32) ss += smem[g * entries + k];
    ss = warp_sum_f32(ss);
    if (lane == 0) rs[g] = 1.f / sqrtf(ss / static_cast<float>(len) + eps);
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    if (i >= cols) continue;
    const float4 w = ld_elem4(norm.w + i);
    const int g = min(i / len, parts - 1);
    if (quad) {
      const float r = rs[g];
      v[j].x *= r * w.x; v[j].y *= r * w.y; v[j].z *= r * w.z; v[j].w *= r * w.w;
    } else {                                               // (weights of padded columns are zero)
      v[j].x *= rs[g] * w.x;
      v[j].y *= rs[min((i + 1) / len, parts - 1)] * w.y;
      v[j].z *= rs[min((i + 2) / len, parts - 1)] * w.z;
      v[j].w *= rs[min((i + 3) / len, parts - 1)] * w.w;
    }
  }
  add_row<NT, NV>(v, norm.b, cols);
}

struct StreamNorm {
  float* x;                  // [rows, cols]
  const float* delta;        // [rows, cols] or null
  const float* delta_b;      // [cols] or null: added to the delta
  const float* vec;          // [cols] or null: added to every row
  float mult, eps;
  RowNorm post, pre;
  int64_t out_stride;
  int cols, n, parts;        // parts: of the norms over parts
};

// PARTS: post and pre are norms over parts, and expert rows may be the input itself.  PAIR: the delta is the sum of two rows.
template <typename T, int NT, int NV, bool PARTS, bool PAIR>
__global__ void __launch_bounds__(NT)
stream_norm_kernel(StreamNorm p, MoeRows<T> moe, SecondRow pair, T* __restrict__ out) {
  extern __shared__ __align__(16) float sn_smem[];         // PARTS: [cols + parts]
  __shared__ float scratch[NT / 32];
  pdl_wait();
  float* __restrict__ x = p.x;
  const float* __restrict__ delta = p.delta;
  const int cols = p.cols, n = p.n;
  const size_t row = blockIdx.x, base = row * cols;
  float4 v[NV];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool add = delta != nullptr || moe.y != nullptr;
  const float sg = moe.gate != nullptr ? sigmoid_f32(moe.gate[row * moe.gate_stride]) : 1.f;
  auto norm = [&](float4 (&u)[NV], const RowNorm& w) {
    if (PARTS && w.kind == kNormParts) norm_parts<NT, NV>(u, w, cols, n, p.parts, p.eps, sn_smem);
    else if (!PARTS) norm_row<NT, NV>(u, w, cols, n, p.eps, scratch);
  };
  if (add) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = (threadIdx.x + NT * j) * 4;
      v[j] = zero;
      if (i >= cols) continue;
      if (delta != nullptr) { v[j] = ld_elem4(delta + base + i); continue; }
      for (int k = 0; k < moe.top; ++k) {
        const int pr = moe.pair_row[row * moe.top + k];
        if (pr < 0) {                                      // the input itself
          if (!PARTS || moe.self == nullptr) continue;
          const float4 a = ld_elem4(moe.self + base + i);
          const float f = moe.wts[row * moe.top + k];
          v[j].x = fmaf(f, a.x, v[j].x); v[j].y = fmaf(f, a.y, v[j].y); v[j].z = fmaf(f, a.z, v[j].z); v[j].w = fmaf(f, a.w, v[j].w);
          continue;
        }
        const float4 a = ld_elem4(moe.y + static_cast<size_t>(pr) * cols + i);
        v[j].x += a.x; v[j].y += a.y; v[j].z += a.z; v[j].w += a.w;
      }
      if (moe.shared != nullptr) {
        const float4 a = ld_elem4(moe.shared + base + i);
        v[j].x = fmaf(sg, a.x, v[j].x); v[j].y = fmaf(sg, a.y, v[j].y); v[j].z = fmaf(sg, a.z, v[j].z); v[j].w = fmaf(sg, a.w, v[j].w);
      }
    }
    add_row<NT, NV>(v, p.delta_b, cols);
    if (PAIR) {
      float4 u[NV];
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int i = (threadIdx.x + NT * j) * 4;
        u[j] = i < cols ? ld_elem4(pair.row + base + i) : zero;
      }
      add_row<NT, NV>(u, pair.bias, cols);
      norm_row<NT, NV>(v, {kNormRms, pair.first_w, nullptr}, cols, n, p.eps, scratch);
      norm_row<NT, NV>(u, {kNormRms, pair.w, nullptr}, cols, n, p.eps, scratch);
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        v[j].x = pair.factor * (v[j].x + u[j].x); v[j].y = pair.factor * (v[j].y + u[j].y);
        v[j].z = pair.factor * (v[j].z + u[j].z); v[j].w = pair.factor * (v[j].w + u[j].w);
      }
    }
    norm(v, p.post);
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    float4 a = i < cols ? ld_elem4(x + base + i) : zero;
    if (add) { a.x = fmaf(p.mult, v[j].x, a.x); a.y = fmaf(p.mult, v[j].y, a.y); a.z = fmaf(p.mult, v[j].z, a.z); a.w = fmaf(p.mult, v[j].w, a.w); }
    v[j] = a;
    if (i < cols && add && p.vec == nullptr) st_elem4(x + base + i, a);
  }
  if (p.vec != nullptr) {
    add_row<NT, NV>(v, p.vec, cols);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = (threadIdx.x + NT * j) * 4;
      if (i < cols) st_elem4(x + base + i, v[j]);
    }
  }
  norm(v, p.pre);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + NT * j) * 4;
    if (i < cols) st_elem4(out + row * p.out_stride + i, v[j]);
  }
}

template <typename T, bool PARTS, bool PAIR>
static int launch_stream_norm(const StreamNorm& p, const MoeRows<T>& moe, const SecondRow& pair, T* out, int rows, cudaStream_t st) {
  const int cols = p.cols;
  const size_t smem = PARTS ? static_cast<size_t>(cols + p.parts) * sizeof(float) : 0;
#define DGPP_SN(NT, NV)                                                                                                              \
  do {                                                                                                                               \
    if (smem > 48 * 1024)                                                                                                            \
      DGPP_CUDA_OK(cudaFuncSetAttribute(stream_norm_kernel<T, NT, NV, PARTS, PAIR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024)); \
    stream_norm_kernel<T, NT, NV, PARTS, PAIR><<<rows, NT, smem, st>>>(p, moe, pair, out);                                           \
  } while (0)
  if (cols <= 1024) DGPP_SN(256, 1);
  else if (cols <= 2048) DGPP_SN(256, 2);
  else if (cols <= 4096) DGPP_SN(256, 4);
  else if (cols <= 8192) DGPP_SN(512, 4);
  else DGPP_SN(1024, 4);
#undef DGPP_SN
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

template <typename T>
static int launch_stream_norm_kind(const StreamNorm& p, const MoeRows<T>& moe, const SecondRow& pair, T* out, int rows, cudaStream_t st) {
  const bool two = pair.row != nullptr;
  if (p.parts > 0) return two ? launch_stream_norm<T, true, true>(p, moe, pair, out, rows, st) : launch_stream_norm<T, true, false>(p, moe, pair, out, rows, st);
  return two ? launch_stream_norm<T, false, true>(p, moe, pair, out, rows, st) : launch_stream_norm<T, false, false>(p, moe, pair, out, rows, st);
}

// grid (parts, rows); y [rows, parts * gp] fp32.  The last part's CTA also clears the columns up to `pad`.
template <typename T, int V>
__global__ void __launch_bounds__(kStreamThreads)
gated_part_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, int64_t z_stride, const float* __restrict__ w,
                       T* __restrict__ out, int64_t out_stride, int gp, int pad, float eps) {
  extern __shared__ __align__(16) float pn_smem[];         // [gp]
  __shared__ float scratch[kStreamThreads / 32];
  pdl_wait();
  const int part = blockIdx.x, n = static_cast<int>(gridDim.x) * gp;
  const size_t row = blockIdx.y;
  const float* yp = y + row * n + static_cast<size_t>(part) * gp;
  const T* zp = z + row * z_stride + static_cast<size_t>(part) * gp;
  T* dst = out + row * out_stride + static_cast<size_t>(part) * gp;
  const float* wp = w + static_cast<size_t>(part) * gp;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < gp; i += kStreamThreads * V) {
    float a[V];
    if (V == 4) {
      const float4 u = ld_elem4(yp + i), g = ld_elem4(zp + i);
      a[0] = u.x * silu_f32(g.x); a[1 % V] = u.y * silu_f32(g.y); a[2 % V] = u.z * silu_f32(g.z); a[3 % V] = u.w * silu_f32(g.w);
    } else {
      a[0] = yp[i] * silu_f32(ld_elem(zp + i));
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      ss = fmaf(a[e], a[e], ss);
      pn_smem[i + e] = a[e];
    }
  }
  const float r = 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(gp) + eps);
  for (int i = threadIdx.x * V; i < gp; i += kStreamThreads * V) {      // a thread reads back what it wrote
    if (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(pn_smem + i), g = ld_elem4(wp + i);
      st_elem4(dst + i, make_float4(a.x * r * g.x, a.y * r * g.y, a.z * r * g.z, a.w * r * g.w));
    } else {
      st_elem(dst + i, pn_smem[i] * r * wp[i]);
    }
  }
  if (part == static_cast<int>(gridDim.x) - 1)
    for (int i = n + threadIdx.x; i < pad; i += kStreamThreads) st_elem(out + row * out_stride + i, 0.f);
}

// gate_up [rows, stride] (TI): gate columns, then up columns, `inter` each.  tiles: rows come in tiles of `bn`, and those whose
// entry is negative are skipped.
template <typename TI, typename T>
__global__ void __launch_bounds__(kStreamThreads)
clamped_glu_kernel(const TI* __restrict__ gate_up, int64_t stride, const float* __restrict__ row_w, const int32_t* __restrict__ tiles, int bn,
                   T* __restrict__ out, int inter, float limit, float alpha, float shift, int weigh_out) {
  pdl_wait();
  const size_t row = blockIdx.y;
  if (tiles != nullptr && tiles[row / bn] < 0) return;
  const int i = (blockIdx.x * kStreamThreads + threadIdx.x) * 8;
  if (i >= inter) return;
  const float w = row_w != nullptr ? row_w[row] : 1.f, s = weigh_out ? 1.f : w, r = weigh_out ? w : 1.f;
  const TI* gp = gate_up + row * stride + i;
  float g[8], u[8];
  ld_elem8(gp, g);
  ld_elem8(gp + inter, u);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    const float a = fminf(g[e] * s, limit), b = fminf(fmaxf(u[e] * s, -limit), limit);
    const float sg = sizeof(T) == 4 ? sigmoid_f32(alpha * a) : __fdividef(1.f, 1.f + __expf(-alpha * a));
    g[e] = r * a * sg * (b + shift);
  }
  st_elem8(out + row * inter + i, g);
}

enum RowAct { kRelu2 = 0, kGeluErf = 1 };

// erf for rows that are rounded to 16 bits (absolute error 1.5e-7): formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical
// Functions.
__device__ __forceinline__ float erf_rows(float x) {
  const float a = fabsf(x), t = __fdividef(1.f, fmaf(0.3275911f, a, 1.f));
  float p = fmaf(1.061405429f, t, -1.453152027f);
  p = fmaf(p, t, 1.421413741f);
  p = fmaf(p, t, -0.284496736f);
  p = fmaf(p, t, 0.254829592f);
  return copysignf(fmaf(-p * t, __expf(-a * a), 1.f), x);
}

// x [rows, stride] (TI) -> out [rows, inter]; tiles: rows come in tiles of `bn`, and those whose entry is negative are skipped.
template <typename TI, typename T, int ACT>
__global__ void __launch_bounds__(kStreamThreads)
act_rows_kernel(const TI* __restrict__ x, int64_t stride, const float* __restrict__ row_w, const int32_t* __restrict__ tiles, int bn,
                T* __restrict__ out, int inter) {
  pdl_wait();
  const size_t row = blockIdx.y;
  if (tiles != nullptr && tiles[row / bn] < 0) return;
  const int i = (blockIdx.x * kStreamThreads + threadIdx.x) * 8;
  if (i >= inter) return;
  const float r = row_w != nullptr ? row_w[row] : 1.f;
  float v[8];
  ld_elem8(x + row * stride + i, v);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    const float z = ACT == kRelu2 ? fmaxf(v[e], 0.f) : v[e];
    const float s = z * 0.70710678118654752f;
    v[e] = r * (ACT == kRelu2 ? z * z : 0.5f * z * (1.f + (sizeof(T) == 4 ? erff(s) : erf_rows(s))));
  }
  st_elem8(out + row * inter + i, v);
}

template <typename T>
__global__ void __launch_bounds__(kStreamThreads)
token_gate_kernel(const float* __restrict__ gate, const int32_t* __restrict__ ids, const T* __restrict__ table, int64_t table_stride, int col,
                  T* __restrict__ out, int dim, int vocab) {
  pdl_wait();
  const size_t row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* e = table + static_cast<size_t>(id) * table_stride + col;
  for (int i = threadIdx.x * 4; i < dim; i += kStreamThreads * 4) {
    const float4 g = ld_elem4(gate + row * dim + i), t = ld_elem4(e + i);
    st_elem4(out + row * dim + i, make_float4(gelu_tanh_f32(g.x) * t.x, gelu_tanh_f32(g.y) * t.y, gelu_tanh_f32(g.z) * t.z, gelu_tanh_f32(g.w) * t.w));
  }
}

__global__ void __launch_bounds__(kStreamThreads) softcap_kernel(float* __restrict__ x, int64_t n, float cap) {
  pdl_wait();
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * kStreamThreads + threadIdx.x; i < n; i += static_cast<int64_t>(gridDim.x) * kStreamThreads)
    x[i] = cap * tanhf(x[i] / cap);
}

}  // namespace dgpp

using namespace dgpp;

// `f32` selects fp32 activations (else bf16) in every entry point below.
// copy: optional second place of the rows, in the activations' type with a row stride of its own.
DGPP_API int dgpp_embed_rows(const void* ids, const void* table, void* out, void* copy, int64_t copy_stride, int rows, int cols, int vocab, float scale,
                             int f32, cudaStream_t st) {
  DGPP_REQUIRE(copy_stride % 8 == 0, "embed_rows: row stride %lld", static_cast<long long>(copy_stride));
  DGPP_REQUIRE(cols % 8 == 0, "embed_rows: %d columns (a multiple of 8)", cols);
  if (rows == 0) return 0;
  if (f32) embed_rows_kernel<float><<<rows, kStreamThreads, 0, st>>>(static_cast<const int32_t*>(ids), static_cast<const float*>(table), static_cast<float*>(out), static_cast<float*>(copy), copy_stride, cols, vocab, scale);
  else embed_rows_kernel<bf16><<<rows, kStreamThreads, 0, st>>>(static_cast<const int32_t*>(ids), static_cast<const bf16*>(table), static_cast<float*>(out), static_cast<bf16*>(copy), copy_stride, cols, vocab, scale);
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

// gate_f32: the gate rows are fp32 although the activations are bf16.  silu: the gate passes silu, else a sigmoid.  den: optional fp32
// [rows, groups], divides o.  w_stride: 0, or columns between the groups' weights.
DGPP_API int dgpp_gated_group_norm(const void* o, const void* den, const void* gate, int64_t gate_stride, const void* w, int w_stride, void* out, int64_t out_stride,
                                   int rows, int groups, int gp, int n, float eps, float scale, int silu, int f32, int gate_f32, cudaStream_t st) {
  DGPP_REQUIRE(gp % 8 == 0 && gate_stride % 8 == 0 && out_stride % 8 == 0 && w_stride % 4 == 0 && n >= 1 && n <= gp, "gated_group_norm: %d of %d columns", n, gp);
  if (rows == 0) return 0;
  const int team = gp <= 512 ? 32 : kStreamThreads;
  const int64_t blocks = dgpp_ceil_div64(static_cast<int64_t>(rows) * groups * team, kStreamThreads);
  const float *op = static_cast<const float*>(o), *wp = static_cast<const float*>(w), *dp = static_cast<const float*>(den);
#define DGPP_GGN(TT, TG) gated_group_norm_kernel<TT, TG><<<static_cast<unsigned>(blocks), kStreamThreads, 0, st>>>( \
      op, dp, static_cast<const TG*>(gate), gate_stride, wp, w_stride, static_cast<TT*>(out), out_stride, rows, groups, gp, n, eps, scale, silu, team)
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

// post / pre: 0 nothing, 1 RMS norm, 2 layer norm, 3 RMS norm over each of `parts` equal parts (then the other one too, or nothing), each with its weights
// and perhaps a bias.  The delta is `delta` (fp32 [rows, cols]), or the expert rows y[pair_row[r * top + j]] (negative: wts[r * top + j]
// times `self`, or nothing) plus sigmoid(gate) * shared (no gate: shared; y, shared, self: activations), or absent; delta_b [cols] is
// added to it.  delta2: the delta is pair_factor * (rms(delta + delta_b) * pair_w1 + rms(delta2 + delta2_b) * pair_w2).  vec [cols]: added to every
// row of x.
DGPP_API int dgpp_stream_norm(void* x, const void* delta, const void* y, const void* pair_row, int top, const void* shared, const void* gate,
                              int64_t gate_stride, const void* self, const void* wts, const void* delta_b, const void* delta2,
                              const void* delta2_b, const void* pair_w1, const void* pair_w2, float pair_factor, const void* vec, float mult, int post,
                              const void* post_w, const void* post_b, int pre, const void* pre_w, const void* pre_b, int parts, void* out,
                              int64_t out_stride, int rows, int cols, int n, float eps, int f32, cudaStream_t st) {
  DGPP_REQUIRE(cols % 8 == 0 && cols <= 16384 && n >= 1 && n <= cols, "stream_norm: %d of %d columns (at most 16384)", n, cols);
  DGPP_REQUIRE(post >= 0 && post <= 3 && pre >= 0 && pre <= 3 && (!post || post_w) && (!pre || pre_w), "stream_norm: norms %d / %d", post, pre);
  DGPP_REQUIRE(!(delta && y) && (!y || (pair_row && top >= 1)) && (!shared || y) && (!gate || shared) && (!self || (y && wts)), "stream_norm: one delta only");
  DGPP_REQUIRE(!delta2 || (delta && pair_w1 && pair_w2), "stream_norm: the second row needs a first one, and weights");
  DGPP_REQUIRE(out_stride % 8 == 0 && out_stride >= cols && (!delta_b || delta || y), "stream_norm: output rows of %lld", static_cast<long long>(out_stride));
  const bool in_parts = post == kNormParts || pre == kNormParts;
  DGPP_REQUIRE(!in_parts || (post % kNormParts == 0 && pre % kNormParts == 0 && parts >= 1 && n % parts == 0),
               "stream_norm: norms %d / %d over %d parts of %d columns", post, pre, parts, n);
  DGPP_REQUIRE(!self || in_parts, "stream_norm: identity experts come with norms over parts (perhaps one)");
  if (rows == 0) return 0;
  auto f = [](const void* q) { return static_cast<const float*>(q); };
  const StreamNorm p = {static_cast<float*>(x), f(delta), f(delta_b), f(vec), mult, eps, {post, f(post_w), f(post_b)}, {pre, f(pre_w), f(pre_b)},
                        out_stride, cols, n, in_parts ? parts : 0};
  const SecondRow pair = {f(delta2), f(delta2_b), f(pair_w2), f(pair_w1), pair_factor};
  const int32_t* pr = static_cast<const int32_t*>(pair_row);
  if (f32) {
    const MoeRows<float> m = {f(y), pr, f(shared), f(gate), gate_stride, f(self), f(wts), top};
    return launch_stream_norm_kind<float>(p, m, pair, static_cast<float*>(out), rows, st);
  }
  auto h = [](const void* q) { return static_cast<const bf16*>(q); };
  const MoeRows<bf16> m = {h(y), pr, h(shared), f(gate), gate_stride, h(self), f(wts), top};
  return launch_stream_norm_kind<bf16>(p, m, pair, static_cast<bf16*>(out), rows, st);
}

DGPP_API int dgpp_gated_part_norm(const void* y, const void* z, int64_t z_stride, const void* w, void* out, int64_t out_stride, int rows,
                                  int parts, int gp, int pad, float eps, int f32, cudaStream_t st) {
  DGPP_REQUIRE(parts >= 1 && gp >= 1 && parts <= 65535 && rows <= 65535, "gated_part_norm: %d parts of %d columns", parts, gp);
  const size_t smem = static_cast<size_t>(gp) * sizeof(float);
  DGPP_REQUIRE(smem <= 200 * 1024, "gated_part_norm: parts of %d columns (at most 51200)", gp);
  if (rows == 0) return 0;
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(gated_part_norm_kernel<bf16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    DGPP_CUDA_OK(cudaFuncSetAttribute(gated_part_norm_kernel<bf16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    DGPP_CUDA_OK(cudaFuncSetAttribute(gated_part_norm_kernel<float, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    DGPP_CUDA_OK(cudaFuncSetAttribute(gated_part_norm_kernel<float, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  const bool wide = gp % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0;
  const float *yp = static_cast<const float*>(y), *wp = static_cast<const float*>(w);
#define DGPP_GPN(TT, V) gated_part_norm_kernel<TT, V><<<dim3(parts, rows), kStreamThreads, smem, st>>>( \
      yp, static_cast<const TT*>(z), z_stride, wp, static_cast<TT*>(out), out_stride, gp, pad, eps)
  if (f32) { if (wide) DGPP_GPN(float, 4); else DGPP_GPN(float, 1); }
  else { if (wide) DGPP_GPN(bf16, 4); else DGPP_GPN(bf16, 1); }
#undef DGPP_GPN
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// in_f32: gate_up is fp32 although the output is bf16.  weigh_out: row_w multiplies the result, else the inputs.
DGPP_API int dgpp_clamped_glu(const void* gate_up, int64_t stride, const void* row_w, const void* tiles, int bn, void* out, int rows, int inter,
                              float limit, float alpha, float shift, int weigh_out, int f32, int in_f32, cudaStream_t st) {
  DGPP_REQUIRE(inter % 8 == 0 && stride % 8 == 0 && bn >= 1, "clamped_glu: width %d (a multiple of 8)", inter);
  if (rows == 0) return 0;
  DGPP_REQUIRE(rows <= 65535, "clamped_glu: %d rows", rows);
  const dim3 grid(dgpp_ceil_div(inter / 8, kStreamThreads), rows);
  const float* rw = static_cast<const float*>(row_w);
  const int32_t* tl = static_cast<const int32_t*>(tiles);
#define DGPP_CG(TI, TT) clamped_glu_kernel<TI, TT><<<grid, kStreamThreads, 0, st>>>(static_cast<const TI*>(gate_up), stride, rw, tl, bn, \
                                                                                   static_cast<TT*>(out), inter, limit, alpha, shift, weigh_out)
  if (f32) DGPP_CG(float, float);
  else if (in_f32) DGPP_CG(float, bf16);
  else DGPP_CG(bf16, bf16);
#undef DGPP_CG
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// act: 0 square of relu, 1 gelu (erf form).  in_f32: x is fp32 although the output is bf16.  row_w [rows] or null multiplies the result.
DGPP_API int dgpp_act_rows(const void* x, int64_t stride, const void* row_w, const void* tiles, int bn, void* out, int rows, int inter, int act, int f32,
                           int in_f32, cudaStream_t st) {
  DGPP_REQUIRE(inter % 8 == 0 && stride % 8 == 0 && bn >= 1 && (act == kRelu2 || act == kGeluErf), "act_rows: width %d (a multiple of 8), activation %d", inter, act);
  if (rows == 0) return 0;
  DGPP_REQUIRE(rows <= 65535, "act_rows: %d rows", rows);
  const dim3 grid(dgpp_ceil_div(inter / 8, kStreamThreads), rows);
  const float* rw = static_cast<const float*>(row_w);
  const int32_t* tl = static_cast<const int32_t*>(tiles);
#define DGPP_AR(TI, TT)                                                                                                                        \
  do {                                                                                                                                         \
    const TI* xp = static_cast<const TI*>(x);                                                                                                  \
    TT* op = static_cast<TT*>(out);                                                                                                            \
    if (act == kRelu2) act_rows_kernel<TI, TT, kRelu2><<<grid, kStreamThreads, 0, st>>>(xp, stride, rw, tl, bn, op, inter);                    \
    else act_rows_kernel<TI, TT, kGeluErf><<<grid, kStreamThreads, 0, st>>>(xp, stride, rw, tl, bn, op, inter);                                \
  } while (0)
  if (f32) DGPP_AR(float, float);
  else if (in_f32) DGPP_AR(float, bf16);
  else DGPP_AR(bf16, bf16);
#undef DGPP_AR
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// gate [rows, dim] fp32; table [vocab, table_stride] in the activations' type, `col`: the layer's first column.
DGPP_API int dgpp_token_gate(const void* gate, const void* ids, const void* table, int64_t table_stride, int col, void* out, int rows, int dim,
                             int vocab, int f32, cudaStream_t st) {
  DGPP_REQUIRE(dim % 8 == 0 && table_stride % 8 == 0 && col % 8 == 0, "token_gate: %d columns from %d", dim, col);
  if (rows == 0) return 0;
  if (f32) token_gate_kernel<float><<<rows, kStreamThreads, 0, st>>>(static_cast<const float*>(gate), static_cast<const int32_t*>(ids), static_cast<const float*>(table), table_stride, col, static_cast<float*>(out), dim, vocab);
  else token_gate_kernel<bf16><<<rows, kStreamThreads, 0, st>>>(static_cast<const float*>(gate), static_cast<const int32_t*>(ids), static_cast<const bf16*>(table), table_stride, col, static_cast<bf16*>(out), dim, vocab);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

DGPP_API int dgpp_softcap(void* x, int64_t n, float cap, cudaStream_t st) {
  DGPP_REQUIRE(cap > 0.f, "softcap: %f", static_cast<double>(cap));
  if (n == 0) return 0;
  const int64_t blocks = dgpp_ceil_div64(n, kStreamThreads);
  softcap_kernel<<<static_cast<unsigned>(blocks > 1184 ? 1184 : blocks), kStreamThreads, 0, st>>>(static_cast<float*>(x), n, cap);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

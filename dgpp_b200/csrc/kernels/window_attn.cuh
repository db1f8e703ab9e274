// GQA over a paged cache of 16-bit or true 32-bit keys and values, of a sliding window, of the row's own chunk of positions, or of
// the whole sequence (a window nobody fills), with a softmax scale of its own and value heads that may be wider or narrower than the
// key heads.
//
//   query head h reads key/value head g = h / (hq / hkv)
//   row at position i attends to positions lo(i) .. i:  p = softmax(scale * q . k),  out = sum p v
//   lo(i) = max(0, i - window + 1), or i - i % window (chunked); the sequence's first keep_first positions are seen from everywhere
//
// What comes before the scores (each part optional, fp32, in this order): biases of q, k and v; a causal depthwise convolution over time
// on every channel of q, k and v; RMS norm of q and k per head or over the whole projection; rotation of the first `rot` columns of a
// head, column i < rot / 2 with column i + rot / 2; a factor on q that grows with the position, 1 + coef * ln(floor((i + 1) / every) + 1).
// Values: an RMS norm per head without weights; rotation of the whole head by the position (halves of the padded width: columns m and
// m + DV / 2), which every output takes back by its own position.  Scores may be capped, cap * tanh(s / cap); a sink per head may stand
// in the softmax's denominator.  Behind them, optional: a sigmoid gate per head.
//
// The convolution's history is a ring of `taps` inputs (bias included) per channel and request, entry p % taps for position p; zeros
// before position 0.  Decode CTAs convolve what they need themselves; prompt rows have been convolved before (short_conv.cu).
//
// Differential attention (maps = 2): a value head has two key heads, and every output head two query heads, whose attentions a1, a2
// over the same values make one output o = a1 - lambda a2, divided by its root mean square, times a factor and a sigmoid gate per
// column.  Query heads are laid out [kv head][map][head of the group], key heads [kv head][map].
//
// The projections of a row sit in one fused row (T = bf16 or fp32); head widths are padded to multiples of 64 with zero
// columns (D for queries / keys, DV for values), `dim` is the true key width that the norms divide by.
// Cache: k [blocks, hkv * maps, page, D], v [blocks, hkv, page, DV].
//
//   qk_norm_append   prompt rows: prepares q in place, appends prepared k and v to the cache (one CTA per row); writes the angles by
//                    which a row's outputs are turned back, for the tensor-core kernel
//   window_attn      one (row, kv head, split of the window) per CTA; `fused` = every row is the newest token of its
//                    request and the CTA prepares q, prepares and appends k / v itself (decode: one launch per layer)
//   diff_combine     the merge of the splits and the combination of the two maps, one warp per (row, head)
// Softmax statistics and sums are fp32; the partials of the splits merge in ascending order.
//
// EXT is the form with any of: a convolution, kept first tokens, a cap, a sink, value norms, rotated values (one map).  window_attn.cu holds
// the entry points of the plain form, window_attn_ext.cu those of the other, so that each family compiles and runs only what it has.
#pragma once
#include <math.h>
#include <string.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"
#include "common/rope.cuh"

namespace dgpp {

struct WindowAttnParams {
  void* proj;               // [rows, stride]: q heads at q_off + h * D, k heads at k_off + g * D, v heads at v_off + g * DV
  int64_t stride;
  int q_off, k_off, v_off;
  const float* wq;          // fp32 norm weights, zero beyond dim: [D], or one row of the whole projection [hq * D] / [hkv * maps * D]
  const float* wk;
  const float *bq, *bk, *bv;  // fp32 biases [hq * D], [hkv * maps * D], [hkv * DV], or null
  const float* freq;        // [2, rot / 2]: rotation frequencies, leading and residual term
  void* k_cache;
  void* v_cache;
  const int32_t* block_table;
  const int32_t* row_req;
  const int32_t* positions;
  const int32_t* row_list;  // optional: the rows of this launch (else 0 .. grid - 1)
  float* part_ml;           // [launch rows, hq, splits, 2]   (splits > 1 or two maps; else null)
  float* part_acc;          // [launch rows, hq, splits, DV]
  void* out;                // [rows, out_stride] head h at column h * DV
  int64_t out_stride;
  int hq, hkv, maps, D, DV, dim, page, max_blocks, splits, window, chunked, fused;
  int norm;                 // 0: none, 1: per head, 2: over the whole projection
  int rot, temp_every, gate_off;   // gate_off: column of the row with the gate of head 0 (negative: no gate)
  float scale, eps, out_scale, temp_coef;
  const float* vfreq;       // [2, DV / 2]: frequencies of rotated values, or null
  float2* turn;             // [rows, DV / 2] cosines and sines of the rows' value angles (qk_norm_append writes them), or null
  const float* conv_w;      // [taps, channels] (last row: the current token), channels q | k | v; null: no convolution here
  float* ring;              // [requests, taps, channels]
  const float* sink;        // [hq] or null
  int vdim, vnorm, taps, keep_first;
  float softcap;            // 0: none
};

// What window_attn takes beyond the common arguments; kept in step with the Python structure that fills it.
struct WindowExtras {
  const float* vfreq;
  float2* turn;
  const float* conv_w;
  float* ring;
  const float* sink;
  int vdim, vnorm, taps, keep_first;
  float softcap;
};

constexpr int kWaWarps = 4;

template <typename T>
__device__ __forceinline__ float wa_exp(float x);
template <>
__device__ __forceinline__ float wa_exp<float>(float x) { return expf(x); }
template <>
__device__ __forceinline__ float wa_exp<bf16>(float x) { return __expf(x); }

__device__ __forceinline__ size_t wa_token(const WindowAttnParams& p, const int32_t* bt, int heads, int g, int t) {
  return (static_cast<size_t>(bt[t / p.page]) * heads + g) * p.page + t % p.page;
}

// cap * tanh(s / cap)
template <typename T>
__device__ __forceinline__ float wa_cap(float s, float cap);
template <>
__device__ __forceinline__ float wa_cap<float>(float s, float cap) { return cap * tanhf(s / cap); }
template <>
__device__ __forceinline__ float wa_cap<bf16>(float s, float cap) {
  return cap - __fdividef(2.f * cap, 1.f + __expf(__fdividef(2.f * s, cap)));
}

// Sum, weights' sum and maximum of a row's keys -> the finished output of one column, the sink included.
template <typename T, bool EXT>
__device__ __forceinline__ float wa_finish(const WindowAttnParams& p, float a, float l, float m, int head) {
  if (EXT && p.sink != nullptr) {
    const float s = p.sink[head], top = fmaxf(m, s), c = m == -INFINITY ? 0.f : wa_exp<T>(m - top);
    a *= c;
    l = l * c + wa_exp<T>(s - top);
  }
  return l > 0.f ? a / l : 0.f;
}

__device__ __forceinline__ float wa_temperature(const WindowAttnParams& p, int pos) {
  return p.temp_coef == 0.f ? 1.f : fmaf(p.temp_coef, logf(static_cast<float>((pos + 1) / p.temp_every) + 1.f), 1.f);
}

// Sum of squares of n columns (bias added), this thread's part.
template <typename T>
__device__ __forceinline__ float wa_squares(const T* src, const float* bias, int n, int first, int step) {
  constexpr int VN = Vec16<T>::N;
  float ss = 0.f;
  for (int c = first * VN; c < n; c += step * VN) {
    float f[VN];
    Vec16<T>::load(src + c, f);
#pragma unroll
    for (int j = 0; j < VN; ++j) {
      const float v = f[j] + (bias != nullptr ? bias[c + j] : 0.f);
      ss = fmaf(v, v, ss);
    }
  }
  return ss;
}

// Cosine and sine of `half` rotated pairs, by the whole CTA (a barrier follows).
__device__ __forceinline__ void wa_angles(const float* freq, int half, int pos, float2* cs) {
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    rope_angle(freq, half, pos, i, sn, c);
    cs[i] = make_float2(c, sn);
  }
}

__device__ __forceinline__ int wa_channels(const WindowAttnParams& p) { return (p.hq + p.hkv * p.maps) * p.D + p.hkv * p.DV; }

// Convolution at position pos of `n` channels from channel ch0 (projection columns src, biases or null) into dst, by the whole CTA; keep:
// the inputs go to the ring.
template <typename T>
__device__ __forceinline__ void wa_conv(const WindowAttnParams& p, const T* src, const float* bias, int ch0, int n, int slot, int pos, bool keep, float* dst) {
  const int C = wa_channels(p), now = pos % p.taps;
  float* ring = p.ring + static_cast<size_t>(slot) * p.taps * C + ch0;
  const float* w = p.conv_w + ch0;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float u = ld_elem(src + c) + (bias != nullptr ? bias[c] : 0.f);
    float acc = w[static_cast<size_t>(p.taps - 1) * C + c] * u;
#pragma unroll 4
    for (int j = 1; j < p.taps; ++j)
      if (j <= pos) acc = fmaf(w[static_cast<size_t>(p.taps - 1 - j) * C + c], ring[static_cast<size_t>(now >= j ? now - j : now - j + p.taps) * C + c], acc);
    if (keep) ring[static_cast<size_t>(now) * C + c] = u;
    dst[c] = acc;
  }
}

// One query, key or (VALUE) value head by one warp: bias, norm (`rstd` of the whole projection, or the head's own), rotation and a factor
// into dst, which may be src (a lane holds both columns of a rotated pair).
template <bool VALUE, typename T, typename D>
__device__ __noinline__ void wa_head(const WindowAttnParams& p, const T* src, const float* bias, const float* w, const float2* cs, float rstd,
                                     float factor, int lane, D* dst) {
  const int norm = VALUE ? p.vnorm : p.norm, width = VALUE ? p.DV : p.D, rot = VALUE ? (p.vfreq != nullptr ? p.DV : 0) : p.rot;
  float r = factor;
  if (norm == 1) r *= 1.f / sqrtf(warp_sum_f32(wa_squares(src, bias, width, lane, 32)) / static_cast<float>(VALUE ? p.vdim : p.dim) + p.eps);
  else if (norm == 2) r *= rstd;
  const bool weigh = !VALUE && norm;
  auto value = [&](int d) { return (ld_elem(src + d) + (bias != nullptr ? bias[d] : 0.f)) * (weigh ? r * w[d] : r); };
  const int half = rot / 2;
#pragma unroll 2
  for (int i = lane; i < half; i += 32) {
    const float a = value(i), b = value(i + half);
    st_elem(dst + i, a * cs[i].x - b * cs[i].y);
    st_elem(dst + i + half, b * cs[i].x + a * cs[i].y);
  }
  int d = rot;
  for (; d % 4 != 0; d += 2)                              // (rot is even)
    if (lane < 2) st_elem(dst + d + lane, value(d + lane));
  for (d += lane * 4; d < width; d += 128) {
    float4 v = ld_elem4(src + d), m = make_float4(r, r, r, r);
    if (bias != nullptr) {
      const float4 e = ld_elem4(bias + d);
      v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
    }
    if (weigh) {
      const float4 e = ld_elem4(w + d);
      m.x *= e.x; m.y *= e.y; m.z *= e.z; m.w *= e.w;
    }
    st_elem4(dst + d, make_float4(v.x * m.x, v.y * m.y, v.z * m.z, v.w * m.w));
  }
}

// src: the head's columns (S: the projection's type, or fp32 behind a convolution, which has added the biases)
template <typename T, typename S>
__device__ __noinline__ void wa_append_key(const WindowAttnParams& p, const S* src, const float* bias, const int32_t* bt, const float2* cs, int g, float rstd,
                                           int pos, int lane) {
  wa_head<false>(p, src, bias, p.norm == 2 ? p.wk + static_cast<size_t>(g) * p.D : p.wk, cs, rstd, 1.f, lane,
                 static_cast<T*>(p.k_cache) + wa_token(p, bt, p.hkv * p.maps, g, pos) * p.D);
}

template <typename T, bool EXT, typename S>
__device__ __forceinline__ void wa_append_value(const WindowAttnParams& p, const S* src, const float* bias, const int32_t* bt, const float2* vcs, int g,
                                                int pos, int lane) {
  T* dst = static_cast<T*>(p.v_cache) + wa_token(p, bt, p.hkv, g, pos) * p.DV;
  if constexpr (EXT) {
    wa_head<true>(p, src, bias, nullptr, vcs, 1.f, 1.f, lane, dst);
  } else {
    for (int d = lane * 4; d < p.DV; d += 128) {
      float4 x = ld_elem4(src + d);
      if (bias != nullptr) {
        const float4 e = ld_elem4(bias + d);
        x.x += e.x; x.y += e.y; x.z += e.z; x.w += e.w;
      }
      st_elem4(dst + d, x);
    }
  }
}

// 1 / root mean square of all query columns (part 0) or all key columns (part 1) of a row, by the whole CTA.
template <typename T>
__device__ __forceinline__ float wa_row_rstd(const WindowAttnParams& p, const T* base, int part, float* scratch) {
  const int heads = part ? p.hkv * p.maps : p.hq;
  const float ss = wa_squares(base + (part ? p.k_off : p.q_off), part ? p.bk : p.bq, heads * p.D, threadIdx.x, blockDim.x);
  return 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(heads * p.dim) + p.eps);
}

// grid (rows)
template <typename T, bool EXT>
__global__ void __launch_bounds__(256) qk_norm_append_kernel(const __grid_constant__ WindowAttnParams p) {
  __shared__ float scratch[8];
  __shared__ float2 cs[128], vcs[EXT ? 128 : 1];
  pdl_wait();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hk = p.hkv * p.maps;
  T* base = static_cast<T*>(p.proj) + static_cast<size_t>(row) * p.stride;
  float rq = 1.f, rk = 1.f;
  if (p.norm == 2) {
    rq = wa_row_rstd(p, base, 0, scratch);
    rk = wa_row_rstd(p, base, 1, scratch);
  }
  const int pos = p.positions[row];
  if (p.rot) wa_angles(p.freq, p.rot / 2, pos, cs);
  const bool turned = EXT && p.vfreq != nullptr;
  if (turned) {
    wa_angles(p.vfreq, p.DV / 2, pos, vcs);
    if (p.turn != nullptr && threadIdx.x < p.DV / 2) p.turn[static_cast<size_t>(row) * (p.DV / 2) + threadIdx.x] = vcs[threadIdx.x];
  }
  if (p.rot || turned) __syncthreads();
  const float temp = wa_temperature(p, pos);
  const int32_t* bt = p.block_table + static_cast<size_t>(p.row_req[row]) * p.max_blocks;
  for (int head = warp; head < p.hq + hk + p.hkv; head += 8) {
    if (head < p.hq) {
      const size_t o = static_cast<size_t>(head) * p.D;
      T* q = base + p.q_off + o;
      wa_head<false>(p, q, p.bq ? p.bq + o : nullptr, p.norm == 2 ? p.wq + o : p.wq, cs, rq, temp, lane, q);
    } else if (head < p.hq + hk) {
      const size_t o = static_cast<size_t>(head - p.hq) * p.D;
      wa_append_key<T>(p, base + p.k_off + o, p.bk ? p.bk + o : nullptr, bt, cs, head - p.hq, rk, pos, lane);
    } else {
      const size_t o = static_cast<size_t>(head - p.hq - hk) * p.DV;
      wa_append_value<T, EXT>(p, base + p.v_off + o, p.bv ? p.bv + o : nullptr, bt, vcs, head - p.hq - hk, pos, lane);
    }
  }
}

template <typename T>
__device__ __forceinline__ float wa_gate(const WindowAttnParams& p, int row, int h) {
  return p.gate_off < 0 ? p.out_scale
                        : p.out_scale * sigmoid_f32(ld_elem(static_cast<const T*>(p.proj) + static_cast<size_t>(row) * p.stride + p.gate_off + h));
}

// grid (hkv * head_chunks, splits, rows).  NG query heads of one kv head per CTA, NG / MAPS of every map; a warp scores 32 keys at a
// time (lane = key), then the lanes take value columns 2 * lane + 64 * j.
template <typename T, int NV, int NG, int MAPS, bool EXT>
__global__ void __launch_bounds__(kWaWarps * 32, EXT && NG == 4 ? 5 : 0) window_attn_kernel(const __grid_constant__ WindowAttnParams p) {
  constexpr int DV = NV * 64, VN = Vec16<T>::N, NGM = NG / MAPS, VU = NV <= 2 ? 8 : 4;
  extern __shared__ __align__(16) float wa_smem[];
  float* q_s = wa_smem;                                   // [NG][D]
  float* red_acc = q_s + NG * p.D;                        // [warps][NG][DV]
  float* kv_s = red_acc + kWaWarps * NG * DV;             // [MAPS][D], [DV]: convolved key and value (fused, with a convolution)
  __shared__ float red_m[kWaWarps][NG], red_l[kWaWarps][NG], scratch[kWaWarps];
  __shared__ float2 cs[128], vcs[EXT ? 128 : 1];
  pdl_wait();
  const int group = p.hq / (p.hkv * MAPS), chunks = (group + NGM - 1) / NGM, hk = p.hkv * MAPS;
  const int kvh = blockIdx.x / chunks, g0 = (blockIdx.x % chunks) * NGM;
  const int split = blockIdx.y, row = p.row_list ? p.row_list[blockIdx.z] : static_cast<int>(blockIdx.z);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[row];
  const int ng = min(NGM, group - g0);
  auto head_of = [&](int i) { return (kvh * MAPS + i / NGM) * group + g0 + min(i % NGM, ng - 1); };
  // keys t_begin .. t_end - 1 of the visible ones, counted from position 0 or (EXT) in order: the kept first ones, then those from `first`
  // on; `skip` positions lie between
  const int first = p.chunked ? pos - pos % p.window : max(0, pos + 1 - p.window);
  const int skip = EXT ? max(0, first - p.keep_first) : 0, kept = EXT && skip > 0 ? p.keep_first : 0;
  const int origin = EXT ? 0 : first, len = pos + 1 - skip;
  int per = (len - origin + p.splits - 1) / p.splits;
  per = (per + kWaWarps * 32 - 1) / (kWaWarps * 32) * (kWaWarps * 32);   // every warp scores as many keys; the last splits may be empty
  const int t_begin = origin + split * per;
  const int t_end = min(len, t_begin + per);
  const int32_t* bt = p.block_table + static_cast<size_t>(p.row_req[row]) * p.max_blocks;
  T* base = static_cast<T*>(p.proj) + static_cast<size_t>(row) * p.stride;
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);

  // the CTA that reads the row's own position appends it (head chunks of one kv head write the same bytes)
  const bool append = p.fused && t_begin < len && t_end == len;
  if (p.fused) {
    float rq = 1.f, rk = 1.f;
    if (p.norm == 2) {
      rq = wa_row_rstd(p, base, 0, scratch);
      if (append) rk = wa_row_rstd(p, base, 1, scratch);
    }
    if (p.rot) wa_angles(p.freq, p.rot / 2, pos, cs);
    if (EXT && p.vfreq != nullptr) wa_angles(p.vfreq, p.DV / 2, pos, vcs);
    const bool conv = EXT && p.conv_w != nullptr;
    if (conv) {                                           // (norms over the whole projection do not come with a convolution)
      const int slot = p.row_req[row];
      for (int i = 0; i < NG; ++i) {
        const int c = head_of(i) * p.D;
        wa_conv(p, base + p.q_off + c, p.bq ? p.bq + c : nullptr, c, p.D, slot, pos, split == 0, q_s + i * p.D);
      }
      if (append) {
        const int ck = kvh * MAPS * p.D, cv = kvh * DV;
        wa_conv(p, base + p.k_off + ck, p.bk ? p.bk + ck : nullptr, p.hq * p.D + ck, MAPS * p.D, slot, pos, g0 == 0, kv_s);
        wa_conv(p, base + p.v_off + cv, p.bv ? p.bv + cv : nullptr, (p.hq + hk) * p.D + cv, DV, slot, pos, g0 == 0, kv_s + MAPS * p.D);
      }
    }
    if (conv || p.rot || (EXT && p.vfreq != nullptr)) __syncthreads();
    const float f = p.scale * wa_temperature(p, pos);
    for (int i = warp; i < NG + (append ? MAPS + 1 : 0); i += kWaWarps) {
      if (i < NG) {
        const size_t o = static_cast<size_t>(head_of(i)) * p.D;
        if (conv) wa_head<false>(p, static_cast<const float*>(q_s + i * p.D), nullptr, p.wq, cs, rq, f, lane, q_s + i * p.D);
        else wa_head<false>(p, base + p.q_off + o, p.bq ? p.bq + o : nullptr, p.norm == 2 ? p.wq + o : p.wq, cs, rq, f, lane, q_s + i * p.D);
      } else if (i < NG + MAPS) {
        const int g = kvh * MAPS + i - NG;
        const size_t o = static_cast<size_t>(g) * p.D;
        if (conv) wa_append_key<T>(p, static_cast<const float*>(kv_s + (i - NG) * p.D), nullptr, bt, cs, g, rk, pos, lane);
        else wa_append_key<T>(p, base + p.k_off + o, p.bk ? p.bk + o : nullptr, bt, cs, g, rk, pos, lane);
      } else {
        if (conv) wa_append_value<T, EXT>(p, static_cast<const float*>(kv_s + MAPS * p.D), nullptr, bt, vcs, kvh, pos, lane);
        else wa_append_value<T, EXT>(p, base + p.v_off + static_cast<size_t>(kvh) * DV, p.bv ? p.bv + kvh * DV : nullptr, bt, vcs, kvh, pos, lane);
      }
    }
  } else {
    if (EXT && p.vfreq != nullptr) wa_angles(p.vfreq, p.DV / 2, pos, vcs);
    for (int i = warp; i < NG; i += kWaWarps) {
      const T* q = base + p.q_off + static_cast<size_t>(head_of(i)) * p.D;
      for (int d = lane; d < p.D; d += 32) q_s[i * p.D + d] = ld_elem(q + d) * p.scale;
    }
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
    const int ts = valid ? t : t_end - 1, tv = EXT && ts >= kept ? ts + skip : ts;
    const size_t tok = wa_token(p, bt, p.hkv, kvh, tv);
    float s[NG];
#pragma unroll
    for (int g = 0; g < NG; ++g) s[g] = 0.f;
#pragma unroll
    for (int m0 = 0; m0 < MAPS; ++m0) {
      const T* kr = kc + (MAPS == 1 ? tok : wa_token(p, bt, hk, kvh * MAPS + m0, tv)) * p.D;
#pragma unroll 4
      for (int c = 0; c < p.D; c += VN) {
        float kf[VN];
        Vec16<T>::load(kr + c, kf);
#pragma unroll
        for (int gm = 0; gm < NGM; ++gm) {
          const int g = m0 * NGM + gm;
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
    }
    if (EXT && p.softcap > 0.f) {
#pragma unroll
      for (int g = 0; g < NG; ++g) s[g] = wa_cap<T>(s[g], p.softcap);
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
    for (int tt = 0; tt < n; tt += VU) {                  // VU keys' values in flight; lanes behind the last key weigh 0
      float2 vf[VU][NV];
#pragma unroll
      for (int u = 0; u < VU; ++u) {
        const size_t vtok = __shfl_sync(0xffffffffu, static_cast<unsigned long long>(tok), tt + u);
        const T* vr = vc + vtok * DV + 2 * lane;
#pragma unroll
        for (int j = 0; j < NV; ++j) vf[u][j] = ld_elem2(vr + 64 * j);
      }
#pragma unroll
      for (int u = 0; u < VU; ++u)
#pragma unroll
        for (int g = 0; g < NG; ++g) {
          const float pg = __shfl_sync(0xffffffffu, pr[g], tt + u);
#pragma unroll
          for (int j = 0; j < NV; ++j) {
            acc[g][2 * j] = fmaf(pg, vf[u][j].x, acc[g][2 * j]);
            acc[g][2 * j + 1] = fmaf(pg, vf[u][j].y, acc[g][2 * j + 1]);
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
  for (int i = threadIdx.x; i < NG * DV; i += blockDim.x) {
    const int g = i / DV, d = i % DV;
    if (g % NGM >= ng) continue;
    float mm = -INFINITY;
    for (int w = 0; w < kWaWarps; ++w) mm = fmaxf(mm, red_m[w][g]);
    const bool back = EXT && p.vfreq != nullptr && p.part_ml == nullptr;        // turned back here: this column with its partner
    const int half = DV / 2, d2 = d < half ? d + half : d - half;
    float ll = 0.f, a = 0.f, b = 0.f;
    for (int w = 0; w < kWaWarps; ++w) {
      const float c = red_m[w][g] == -INFINITY ? 0.f : wa_exp<T>(red_m[w][g] - mm);
      ll += red_l[w][g] * c;
      a += red_acc[(w * NG + g) * DV + d] * c;
      if (back) b += red_acc[(w * NG + g) * DV + d2] * c;
    }
    const int h = head_of(g);
    if (back) {
      const float2 cs2 = vcs[d < half ? d : d2];
      a = d < half ? a * cs2.x + b * cs2.y : a * cs2.x - b * cs2.y;
    }
    if (p.part_ml == nullptr) {
      st_elem(static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_stride + static_cast<size_t>(h) * DV + d,
              wa_finish<T, EXT>(p, a, ll, mm, h) * wa_gate<T>(p, row, h));
    } else {
      const size_t pi = (static_cast<size_t>(blockIdx.z) * p.hq + h) * p.splits + split;
      p.part_acc[pi * DV + d] = a;
      if (d == 0) { p.part_ml[pi * 2] = mm; p.part_ml[pi * 2 + 1] = ll; }
    }
  }
}

// grid (hq, rows), DV threads
template <typename T, bool EXT>
__global__ void __launch_bounds__(256) window_attn_combine_kernel(WindowAttnParams p) {
  pdl_wait();
  const int row = p.row_list ? p.row_list[blockIdx.y] : static_cast<int>(blockIdx.y);
  const int h = blockIdx.x, d = threadIdx.x;
  const size_t rh = static_cast<size_t>(blockIdx.y) * p.hq + h;
  float mm = -INFINITY;
  for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.part_ml[(rh * p.splits + s) * 2]);
  float ll = 0.f, a = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float ms = p.part_ml[(rh * p.splits + s) * 2];
    const float c = ms == -INFINITY ? 0.f : wa_exp<T>(ms - mm);
    ll += p.part_ml[(rh * p.splits + s) * 2 + 1] * c;
    a += p.part_acc[(rh * p.splits + s) * p.DV + d] * c;
  }
  if (EXT && p.vfreq != nullptr) {
    __shared__ float both[256];
    const int half = p.DV / 2, m = d < half ? d : d - half;
    both[d] = a;
    __syncthreads();
    float sn, c;
    rope_angle(p.vfreq, half, p.positions[row], m, sn, c);
    a = d < half ? a * c + both[d + half] * sn : a * c - both[m] * sn;
  }
  st_elem(static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_stride + static_cast<size_t>(h) * p.DV + d,
          wa_finish<T, EXT>(p, a, ll, mm, h) * wa_gate<T>(p, row, h));
}

template <typename T, int NV, int NG, int MAPS, bool EXT>
static int launch_wa(const WindowAttnParams& p, int rows, cudaStream_t st) {
  const int chunks = dgpp_ceil_div(p.hq / (p.hkv * MAPS), NG / MAPS);
  const size_t smem = (static_cast<size_t>(NG) * p.D + static_cast<size_t>(kWaWarps) * NG * NV * 64 + (p.conv_w != nullptr ? MAPS * p.D + NV * 64 : 0)) * sizeof(float);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(window_attn_kernel<T, NV, NG, MAPS, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    attr = true;
  }
  window_attn_kernel<T, NV, NG, MAPS, EXT><<<dim3(p.hkv * chunks, p.splits, rows), kWaWarps * 32, smem, st>>>(p);
  DGPP_CUDA_OK(cudaGetLastError());
  if (MAPS == 1 && p.splits > 1) {
    window_attn_combine_kernel<T, EXT><<<dim3(p.hq, rows), NV * 64, 0, st>>>(p);
    DGPP_CUDA_OK(cudaGetLastError());
  }
  return 0;
}

template <typename T, int NV, bool EXT>
static int launch_wa_g(const WindowAttnParams& p, int rows, cudaStream_t st) {
  const int g = p.hq / (p.hkv * p.maps);
  if constexpr (!EXT) {
    if (p.maps == 2) {
      if (g == 1) return launch_wa<T, NV, 2, 2, false>(p, rows, st);
      if (g == 2) return launch_wa<T, NV, 4, 2, false>(p, rows, st);
      return launch_wa<T, NV, 8, 2, false>(p, rows, st);
    }
  }
  if (g == 1) return launch_wa<T, NV, 1, 1, EXT>(p, rows, st);
  if (g == 2) return launch_wa<T, NV, 2, 1, EXT>(p, rows, st);
  if (g <= 4) return launch_wa<T, NV, 4, 1, EXT>(p, rows, st);
  return launch_wa<T, NV, 8, 1, EXT>(p, rows, st);
}

template <typename T, bool EXT>
static int launch_wa_v(const WindowAttnParams& p, int rows, cudaStream_t st) {
  if (p.DV == 64) return launch_wa_g<T, 1, EXT>(p, rows, st);
  if (p.DV == 128) return launch_wa_g<T, 2, EXT>(p, rows, st);
  if (p.DV == 192) return launch_wa_g<T, 3, EXT>(p, rows, st);
  return launch_wa_g<T, 4, EXT>(p, rows, st);
}

static int wa_check(const WindowAttnParams& p, int rows) {
  DGPP_REQUIRE((p.maps == 1 || p.maps == 2) && p.hkv > 0 && p.hq % (p.hkv * p.maps) == 0, "window_attn: %d query heads over %d x %d key heads", p.hq, p.hkv, p.maps);
  DGPP_REQUIRE(p.norm >= 0 && p.norm <= 2 && (!p.norm || (p.wq && p.wk)), "window_attn: norm %d needs its weights", p.norm);
  DGPP_REQUIRE(p.rot >= 0 && p.rot % 2 == 0 && p.rot <= p.dim && (p.rot == 0 || p.freq), "window_attn: %d of %d columns rotated", p.rot, p.dim);
  DGPP_REQUIRE(p.temp_coef == 0.f || p.temp_every >= 1, "window_attn: temperature every %d", p.temp_every);
  DGPP_REQUIRE(p.D % 64 == 0 && p.D >= 64 && p.D <= 256 && p.DV % 64 == 0 && p.DV >= 64 && p.DV <= 256,
               "window_attn: head widths %d / %d (padded to multiples of 64, at most 256)", p.D, p.DV);
  DGPP_REQUIRE(p.stride % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 && p.v_off % 8 == 0, "window_attn: unaligned projection rows");
  DGPP_REQUIRE(p.window >= 1 && p.splits >= 1 && p.page >= 1 && p.dim >= 1 && p.dim <= p.D, "window_attn: window %d splits %d", p.window, p.splits);
  DGPP_REQUIRE(p.part_ml ? p.part_acc != nullptr : p.splits == 1, "window_attn: scratch required when splits > 1");
  DGPP_REQUIRE(rows >= 0 && rows <= 65535, "window_attn: %d rows", rows);
  DGPP_REQUIRE(!p.conv_w || (p.ring && p.taps >= 1 && p.norm != 2), "window_attn: a convolution of %d taps before norm %d", p.taps, p.norm);
  DGPP_REQUIRE(!p.vnorm || (p.vdim >= 1 && p.vdim <= p.DV), "window_attn: value norm over %d of %d columns", p.vdim, p.DV);
  DGPP_REQUIRE(p.keep_first >= 0 && (!p.chunked || p.keep_first == 0) && p.softcap >= 0.f, "window_attn: %d kept tokens, cap %f", p.keep_first, static_cast<double>(p.softcap));
  return 0;
}

}  // namespace dgpp

// What every entry point takes: see WindowAttnParams.  bq / bk / bv, freq (rot = 0), the norm weights (norm = 0) and `extras` (a
// WindowExtras on the host) may be null.
#define WA_COMMON                                                                                                                      \
  void *proj, int64_t stride, int q_off, int k_off, int v_off, const void *wq, const void *wk, const void *bq, const void *bk,          \
      const void *bv, const void *freq, void *k_cache, void *v_cache, const void *block_table, const void *row_req,                    \
      const void *positions, int rows, int hq, int hkv, int maps, int D, int DV, int dim, int page, int max_blocks, int norm, int rot,  \
      int temp_every, float temp_coef, float eps, const void* extras

namespace dgpp {

static WindowAttnParams wa_params(WA_COMMON) {
  WindowAttnParams p;
  memset(&p, 0, sizeof(p));
  p.proj = proj; p.stride = stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  auto f = [](const void* q) { return static_cast<const float*>(q); };
  p.wq = f(wq); p.wk = f(wk); p.bq = f(bq); p.bk = f(bk); p.bv = f(bv); p.freq = f(freq);
  p.k_cache = k_cache; p.v_cache = v_cache;
  p.block_table = static_cast<const int32_t*>(block_table);
  p.row_req = static_cast<const int32_t*>(row_req);
  p.positions = static_cast<const int32_t*>(positions);
  p.hq = hq; p.hkv = hkv; p.maps = maps; p.D = D; p.DV = DV; p.dim = dim; p.page = page; p.max_blocks = max_blocks;
  p.norm = norm; p.rot = rot; p.temp_every = temp_every; p.temp_coef = temp_coef; p.eps = eps;
  if (extras != nullptr) {
    const WindowExtras& x = *static_cast<const WindowExtras*>(extras);
    p.vfreq = x.vfreq; p.turn = x.turn; p.conv_w = x.conv_w; p.ring = x.ring; p.sink = x.sink;
    p.vdim = x.vdim; p.vnorm = x.vnorm; p.taps = x.taps; p.keep_first = x.keep_first; p.softcap = x.softcap;
  }
  p.splits = 1; p.window = 1; p.scale = 1.f; p.out_scale = 1.f; p.gate_off = -1;
  return p;
}
#define WA_ARGS                                                                                                                   \
  proj, stride, q_off, k_off, v_off, wq, wk, bq, bk, bv, freq, k_cache, v_cache, block_table, row_req, positions, rows, hq, hkv, maps, D, \
      DV, dim, page, max_blocks, norm, rot, temp_every, temp_coef, eps, extras

template <bool EXT>
static int wa_append_rows(WA_COMMON, int f32, cudaStream_t st) {
  const WindowAttnParams p = wa_params(WA_ARGS);
  if (wa_check(p, rows)) return -1;
  DGPP_REQUIRE(!p.conv_w, "qk_norm_append: prompt rows are convolved before");
  if (rows == 0) return 0;
  if (f32) qk_norm_append_kernel<float, EXT><<<rows, 256, 0, st>>>(p);
  else qk_norm_append_kernel<bf16, EXT><<<rows, 256, 0, st>>>(p);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// rows: rows of this launch (row_list, int32, names them when given).  fused: see the header.  out_scale multiplies the
// outputs before they are rounded.  part_ml / part_acc: rows * hq * splits * (2 | DV) floats; with two maps they are the result (null
// out), which `dgpp_diff_combine` finishes.
#define WA_ATTEND                                                                                                                  \
  const void *row_list, void *part_ml, void *part_acc, void *out, int64_t out_stride, int splits, int window, int chunked, int fused, \
      int gate_off, float scale, float out_scale, int f32, cudaStream_t st
#define WA_ATTEND_ARGS row_list, part_ml, part_acc, out, out_stride, splits, window, chunked, fused, gate_off, scale, out_scale, f32, st

template <bool EXT>
static int wa_attend_rows(WA_COMMON, WA_ATTEND) {
  WindowAttnParams p = wa_params(WA_ARGS);
  p.row_list = static_cast<const int32_t*>(row_list);
  p.part_ml = static_cast<float*>(part_ml); p.part_acc = static_cast<float*>(part_acc);
  p.out = out; p.out_stride = out_stride;
  p.splits = splits; p.window = window; p.chunked = chunked; p.fused = fused; p.gate_off = gate_off; p.scale = scale; p.out_scale = out_scale;
  if (wa_check(p, rows)) return -1;
  DGPP_REQUIRE(!p.conv_w || p.fused, "window_attn: prompt rows are convolved before");
  DGPP_REQUIRE(maps == 1 ? out != nullptr && (splits > 1) == (part_ml != nullptr) : part_ml != nullptr, "window_attn: no place for the result");
  if (rows == 0) return 0;
  return f32 ? launch_wa_v<float, EXT>(p, rows, st) : launch_wa_v<bf16, EXT>(p, rows, st);
}

}  // namespace dgpp

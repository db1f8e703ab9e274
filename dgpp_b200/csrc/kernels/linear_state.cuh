// Linear-attention layers whose memory is one fp32 matrix S [DK, DV] per head and request:
//
//   channel delta rule   S <- g_t * S (a decay per key channel);  u = b_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
//                        q, k, v pass a causal depthwise convolution and silu, q and k become unit vectors, q is scaled;
//                        g_t = exp(-exp(A) softplus(a_t + dt)),  b_t = sigmoid(beta_t)
//   scalar delta rule    the same with one decay per token and head, g_t = exp(-exp(A_h) softplus(a_t + dt_h)); its output gate is a
//                        silu of plain columns of the projection
//   lightning            S <- d_h * S + k_t v_t^T (a constant decay per head);  o_t = S^T q_t;  q, k, v = silu(projection)
//   state space          S <- a_t S + dt_t k_t v_t^T (a decay per token and head);  o_t = S^T q_t + D_h v_t
//                        q, k (shared by groups of heads), v pass a causal depthwise convolution with bias and silu;
//                        dt_t = softplus(raw step + bias),  a_t = exp(-exp(A) dt_t)
//   matrix memory        S <- d_t S + w_t k_t v_t^T,  n <- d_t n + w_t k_t,  o_t = S^T q_t / (max(|n . q_t|, exp(-m_t)) + 1e-6)
//                        (the mLSTM of xLSTM); log gates i = cap tanh((raw + bias) / cap), f = logsigmoid(cap tanh((raw + bias) / cap)),
//                        running maximum m_t = max(f + m_(t-1), i) from m = 0, d_t = exp(f + m_(t-1) - m_t), w_t = exp(i - m_t);
//                        a norm per head and a sigmoid gate per column behind it; q, k, v as projected, q scaled
//
// All are one kernel family (template parameter RULE; linear_state.cu, state_space.cu, gated_delta.cu and matrix_memory.cu hold the entry
// points).  A pass
// carries runs of consecutive tokens of any number of requests:
// run r = rows [run_start[r], run_start[r + 1]) of the request in state slot row_slot[first row].
//
//   lin_decode   runs of one token: convolution, norms, gates, state update and read-out of a (row, head) in one CTA with
//                the whole S in registers; the delta rule's output norm and gate are fused in as well
//   lin_prep     token-parallel part of longer runs -> fp32 scratch (unit q / k, v, decays, strengths); ssd_prep: the same for the
//                rules with scalar decays, convolution windows in registers
//   lin_block    16-token blocks in parallel: the block's decay products and token-pair matrices (ssd_block, gated_block:
//                the same for scalar decays, which leave q and k as they are, shared by a group of heads)
//   lin_scan     block-sequential part: one CTA per (32 state columns, head, run), S in registers, the next block's operands
//                streaming in with cp.async while the current one is consumed.  Matrix memory: one more warp of a head's first CTA
//                carries n as the state's column for a value that is always one, and finishes the denominators
//   lin_tail     the newest inputs of the convolution go to the request's ring after every reader is done
//
// The decode kernel takes o_t as (g S)^T q + (k . q) u, the read-out after the write, so both reductions over the key channels
// run together.  A request's first token (position 0) starts from S = 0 and from zeros before it: a slot needs no clearing
// between requests.  The convolution's history is a ring of `taps` inputs per channel, entry p % taps for position p: a
// token never overwrites an entry that its own window reads, so decode CTAs of heads that share key heads do not race.
#pragma once
#include <math.h>
#include <string.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

enum LinearRule { kLightning = 0, kDelta = 1, kStateSpace = 2, kScalarDelta = 3, kMatrix = 4 };

__host__ __device__ constexpr bool is_delta(int rule) { return rule == kDelta || rule == kScalarDelta; }
__host__ __device__ constexpr bool scalar_decay(int rule) { return rule == kStateSpace || rule == kScalarDelta || rule == kMatrix; }

struct LinearArgs {
  const void* proj;         // [rows, stride] (T): conv channels q (hk * DK) | k (hk * DK) | v (hv * DV) from column c_off
  int64_t stride;
  int c_off, b_off;         // b_off: raw write strengths (delta) or raw step sizes (state space) [hv]
  int a_off, g_off;         // raw decays [hv], raw output gates [hv * DV] (scalar delta)
  const float* low;         // [rows, low_stride] fp32: raw decays [hv * DK], then raw output gates [hv * DV] (delta)
  int64_t low_stride;
  const float* conv_w;      // [taps, C] (last row: the current token); null: no convolution
  const float* conv_b;      // [C] or null
  float* ring;              // [slots, taps, C]
  const float* A_log;       // [hv]
  const float* dt_bias;     // [hv * DK] (channel delta), [hv] (state space, scalar delta)
  const float* skip;        // [hv] D (state space)
  const float* decay;       // [hv] (lightning)
  float* state;             // [slots, hv, DK, DV]
  const int32_t* row_slot;  // [rows]
  const int32_t* positions; // [rows]
  const int32_t* run_start; // [runs + 1]
  const int32_t* row_run0;  // [rows] first row of the row's run
  float* prep;              // scratch (see lin_prep)
  float* o;                 // [rows, hv * ow] fp32 read-outs (scan; lightning and state-space decode)
  void* out;                // [rows, out_stride] (T): normed and gated read-outs (delta decode)
  int64_t out_stride;
  const float* norm_w;      // [DV] (matrix memory: [hv * DV])
  float* nstate;            // [slots, hv, DK + 4]: n, then the running maximum m (matrix memory)
  float* den;               // [rows, hv] denominators of the read-outs in `o` (matrix memory)
  const float *i_bias, *f_bias;   // [hv]; raw input gates at b_off, raw forget gates at a_off (matrix memory)
  float gate_cap;
  int rows, runs, blocks, hk, hv, taps, vdim, ow;   // ow: columns of a head's read-out in `o` (DV; state space: vdim)
  float q_scale, eps;
};

template <int DK, int DV>
struct LinGeom {
  static constexpr int kRaw = DK * DV / 64;
  static constexpr int kThreads = kRaw < 128 ? 128 : kRaw;      // at most 1024 (256 x 256)
  static constexpr int kCols4 = DV / 4;
  static constexpr int kParts = kThreads / kCols4;              // threads that share a column
  static constexpr int kPer = DK / kParts;                      // state rows per thread
};

// Convolution of one channel at position pos: w[taps - 1] x + sum_j w[taps - 1 - j] past(j).  The loads of four taps are in
// flight together.  `rows_back` inputs before this one are rows of the pass (x - j * stride), older ones sit in the ring.
template <typename T>
__device__ __forceinline__ float conv_channel(const LinearArgs& a, const T* x, int64_t stride, float xv, int rows_back, int C, int slot,
                                              int pos, int base, int ch) {
  const float* w0 = a.conv_w + static_cast<size_t>(a.taps - 1) * C + ch;
  float acc = a.conv_b != nullptr ? fmaf(*w0, xv, a.conv_b[ch]) : *w0 * xv;
  if (rows_back >= a.taps - 1) {                 // the usual place in a prompt: every past input is a row of the pass
#pragma unroll 3
    for (int j = 1; j < a.taps; ++j) {
      w0 -= C;
      x -= stride;
      acc = fmaf(*w0, ld_elem(x), acc);
    }
    return acc;
  }
  const float* ring = a.ring + static_cast<size_t>(slot) * a.taps * C + ch;
  for (int j0 = 1; j0 < a.taps; j0 += 4) {
    float past[4], w[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = j0 + e;
      past[e] = 0.f;
      w[e] = 0.f;
      if (j < a.taps && j <= pos) {
        w[e] = a.conv_w[static_cast<size_t>(a.taps - 1 - j) * C + ch];
        if (j <= rows_back) past[e] = ld_elem(x - j * stride);
        else past[e] = ring[static_cast<size_t>(base - j + (base < j ? a.taps : 0)) * C];
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) acc = fmaf(w[e], past[e], acc);
  }
  return acc;
}

// Log gates of a row and head (matrix memory).
template <typename T>
__device__ __forceinline__ float2 matrix_gates(const LinearArgs& a, int row, int h) {
  const T* x = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + h;
  const float i = a.gate_cap * tanhf((ld_elem(x + a.b_off) + a.i_bias[h]) / a.gate_cap);
  const float f = a.gate_cap * tanhf((ld_elem(x + a.a_off) + a.f_bias[h]) / a.gate_cap);
  return make_float2(i, -softplus_f32(-f));
}

__device__ __forceinline__ float matrix_den(float nq, float floor) { return fmaxf(fabsf(nq), floor) + 1e-6f; }

__device__ __forceinline__ float4 fma4(float4 s, float a, float4 acc) {
  acc.x = fmaf(s.x, a, acc.x); acc.y = fmaf(s.y, a, acc.y); acc.z = fmaf(s.z, a, acc.z); acc.w = fmaf(s.w, a, acc.w);
  return acc;
}

// grid (hv, rows)
template <typename T, int DK, int DV, int RULE>
__global__ void __launch_bounds__(LinGeom<DK, DV>::kThreads) lin_decode_kernel(LinearArgs a) {
  constexpr bool DELTA = is_delta(RULE), CH = RULE == kDelta, SSD = RULE == kStateSpace, MAT = RULE == kMatrix;
  using G = LinGeom<DK, DV>;
  constexpr int NT = G::kThreads, PER = G::kPer, PARTS = G::kParts;
  extern __shared__ __align__(16) float ld_smem[];
  float* red_n = ld_smem;                                 // [PARTS][DV]
  float* red_m = red_n + PARTS * DV;                      // [PARTS][DV] (delta)
  __shared__ float qs[DK], ks[DK], gs[DK];
  __shared__ __align__(16) float vs[DV], us[DV];
  __shared__ float scal[3];                               // |q|^2 (matrix memory: n . q), |k|^2, q . k
  __shared__ float scratch[32];
  pdl_wait();
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
  const int slot = a.row_slot[row], pos = a.positions[row];
  const int ratio = a.hv / a.hk, hk = h / ratio;
  const int C = 2 * a.hk * DK + a.hv * DV;
  const int cg = tid % G::kCols4, part = tid / G::kCols4;
  float4* sp = reinterpret_cast<float4*>(a.state + (static_cast<size_t>(slot) * a.hv + h) * DK * DV) + cg;
  float4 s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) s[i] = pos > 0 ? sp[static_cast<size_t>(part + PARTS * i) * G::kCols4] : make_float4(0.f, 0.f, 0.f, 0.f);
  // ---- inputs of this head
  const int base = a.conv_w != nullptr ? pos % a.taps : 0;       // this token's ring entry
  const T* x = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.c_off;
#pragma unroll 2
  for (int c = tid; c < 2 * DK + DV; c += NT) {
    const int ch = c < DK ? hk * DK + c : (c < 2 * DK ? (a.hk + hk) * DK + c - DK : 2 * a.hk * DK + h * DV + c - 2 * DK);
    const float xv = ld_elem(x + ch);
    float acc = xv;
    if (a.conv_w != nullptr) {
      acc = conv_channel(a, x + ch, a.stride, xv, 0, C, slot, pos, base, ch);
      if (c >= 2 * DK || h % ratio == 0) a.ring[(static_cast<size_t>(slot) * a.taps + base) * C + ch] = xv;
    }
    if (!MAT) acc = silu_f32(acc);
    if (c < DK) qs[c] = acc;
    else if (c < 2 * DK) ks[c - DK] = acc;
    else vs[c - 2 * DK] = acc;
  }
  float beta = 1.f, dh = 1.f, skip = 0.f, m_new = 0.f;
  float* ns = MAT ? a.nstate + (static_cast<size_t>(slot) * a.hv + h) * (DK + 4) : nullptr;
  if (MAT) {
    const float2 g = matrix_gates<T>(a, row, h);
    const float past = g.y + (pos > 0 ? ns[DK] : 0.f);
    m_new = fmaxf(past, g.x);
    dh = expf(past - m_new);
    beta = expf(g.x - m_new);
  }
  if (SSD) {
    beta = softplus_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.b_off + h) + a.dt_bias[h]);
    dh = expf(-expf(a.A_log[h]) * beta);
    skip = a.skip[h];
  } else if (RULE == kLightning) {
    dh = a.decay[h];
  }
  if (DELTA) {
    const float ea = -expf(a.A_log[h]);
    if (CH) {
      const float* ar = a.low + static_cast<size_t>(row) * a.low_stride + h * DK;
      for (int c = tid; c < DK; c += NT) gs[c] = expf(ea * softplus_f32(ar[c] + a.dt_bias[h * DK + c]));
    } else {
      dh = expf(ea * softplus_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.a_off + h) + a.dt_bias[h]));
    }
    beta = sigmoid_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.b_off + h));
  }
  __syncthreads();
  if (tid < 32) {
    float q2 = 0.f, k2 = 0.f, qk = 0.f, nq = 0.f;
    for (int c = tid; c < DK; c += 32) {
      q2 = fmaf(qs[c], qs[c], q2);
      k2 = fmaf(ks[c], ks[c], k2);
      qk = fmaf(qs[c], ks[c], qk);
      if (MAT) {
        const float n = fmaf(beta, ks[c], pos > 0 ? dh * ns[c] : 0.f);
        ns[c] = n;
        nq = fmaf(n, qs[c], nq);
      }
    }
    if (MAT) nq = warp_sum_f32(nq);
    q2 = warp_sum_f32(q2); k2 = warp_sum_f32(k2); qk = warp_sum_f32(qk);
    if (tid == 0) {
      scal[0] = MAT ? nq : q2; scal[1] = k2; scal[2] = qk;
      if (MAT) ns[DK] = m_new;
    }
  }
  // ---- decay, both reductions
  float4 n4 = make_float4(0.f, 0.f, 0.f, 0.f), m4 = n4;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int r = part + PARTS * i;
    const float g = CH ? gs[r] : dh;
    s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
    n4 = fma4(s[i], qs[r], n4);
    if (DELTA) m4 = fma4(s[i], ks[r], m4);
  }
  *reinterpret_cast<float4*>(red_n + part * DV + 4 * cg) = n4;
  if (DELTA) *reinterpret_cast<float4*>(red_m + part * DV + 4 * cg) = m4;
  __syncthreads();
  const float rq = DELTA ? a.q_scale / sqrtf(scal[0] + 1e-6f) : (MAT ? a.q_scale : 1.f), rk = DELTA ? 1.f / sqrtf(scal[1] + 1e-6f) : 1.f;
  const float qk = scal[2] * rq * rk;
  const float inv = MAT ? 1.f / matrix_den(scal[0] * rq, expf(-m_new)) : 1.f;
  float ss = 0.f;
  for (int c = tid; c < DV; c += NT) {
    float n = 0.f, m = 0.f;
#pragma unroll
    for (int w = 0; w < PARTS; ++w) {
      n += red_n[w * DV + c];
      if (DELTA) m += red_m[w * DV + c];
    }
    const float u = DELTA ? beta * (vs[c] - m * rk) : (SSD || MAT ? beta * vs[c] : vs[c]);
    const float o = (n * rq + qk * u + (SSD ? skip * vs[c] : 0.f)) * inv;
    us[c] = u * rk;                              // the key's norm rides on u
    ss = fmaf(o, o, ss);
    if (DELTA || MAT) vs[c] = o;
    else if (c < a.ow) a.o[(static_cast<size_t>(row) * a.hv + h) * a.ow + c] = o;
  }
  __syncthreads();
  const float4 u4 = *reinterpret_cast<const float4*>(us + 4 * cg);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int r = part + PARTS * i;
    sp[static_cast<size_t>(r) * G::kCols4] = fma4(u4, ks[r], s[i]);
  }
  if (DELTA || MAT) {
    const float r = 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(a.vdim) + a.eps);
    T* dst = static_cast<T*>(a.out) + static_cast<size_t>(row) * a.out_stride + h * DV;
    if (MAT) {
      const T* gt = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.g_off + h * DV;
      for (int c = tid; c < DV; c += NT) st_elem(dst + c, vs[c] * r * a.norm_w[h * DV + c] * sigmoid_f32(ld_elem(gt + c)));
    } else if (CH) {
      const float* gt = a.low + static_cast<size_t>(row) * a.low_stride + a.hv * DK + h * DV;
      for (int c = tid; c < DV; c += NT) st_elem(dst + c, vs[c] * r * a.norm_w[c] * sigmoid_f32(gt[c]));
    } else {
      const T* gt = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.g_off + h * DV;
      for (int c = tid; c < DV; c += NT) st_elem(dst + c, vs[c] * r * a.norm_w[c] * silu_f32(ld_elem(gt + c)));
    }
  }
}

// Scratch of a pass over runs (fp32): per row q, k [hk, DK], v [hv, DV], decays [hv, DK] (delta; lin_block replaces them by
// K * gamma), Q * gamma and the suffix-weighted keys [hv, DK]; per block gamma_16 [hv, DK], P and (delta) T B [hv, 16, 16]; the
// strengths [rows, hv] (delta) at the end.  State space: per row q, k, v, decay and step [hv] each; per block and head P with the
// steps and the skip folded in [16, 16] and 16 prefix products, then 16 write weights.  Scalar delta: per row q, k (not yet unit
// vectors), v, decay and strength; per block and head P and T B [16, 16], then 16 factors each of Q S, of the writes and of K S, and
// gamma_16; the lengths of q and k ride in all of these.  Matrix memory: as state space (d_t and w_t for decay and step), then exp(-m_t)
// [rows, hv].
struct PrepView {
  float *q, *k, *v, *g, *kt, *qt, *kh, *gam, *pm, *tb, *b, *fl;
};
template <int DK, int DV, int RULE>
__device__ __forceinline__ PrepView prep_view(const LinearArgs& a) {
  constexpr bool DELTA = RULE == kDelta;              // (the scalar rule has its own layout)
  PrepView p;
  const size_t R = a.rows, B = a.blocks;
  p.q = a.prep;
  p.k = p.q + R * a.hk * DK;
  p.v = p.k + R * a.hk * DK;
  p.g = p.v + R * a.hv * DV;
  if (scalar_decay(RULE)) {
    p.pm = p.g;
    p.tb = p.pm + B * a.hv * 256;
    p.gam = RULE == kScalarDelta ? p.tb + B * a.hv * 256 : p.tb;
    p.g = p.gam + B * a.hv * (RULE == kScalarDelta ? 64 : 32);
    p.b = p.g + R * a.hv;
    p.kt = p.qt = p.kh = nullptr;
    p.fl = p.b + R * a.hv;
    return p;
  }
  p.fl = nullptr;
  p.kt = p.g;
  p.qt = p.g + (DELTA ? R * a.hv * DK : 0);
  p.kh = p.qt + R * a.hv * DK;
  p.gam = p.kh + R * a.hv * DK;
  p.pm = p.gam + B * a.hv * DK;
  p.tb = p.pm + B * a.hv * 256;
  p.b = p.tb + (DELTA ? B * a.hv * 256 : 0);
  return p;
}

// One warp per (row, unit): units < hk prepare a key head, the others a value head.
template <typename T, int DK, int DV, int RULE>
__global__ void __launch_bounds__(256) lin_prep_kernel(LinearArgs a) {
  constexpr bool DELTA = RULE == kDelta;
  pdl_wait();
  const int lane = threadIdx.x & 31, units = a.hk + a.hv;
  const int warp = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (warp >= a.rows * units) return;
  const int row = warp / units, unit = warp % units;
  const int slot = a.row_slot[row], pos = a.positions[row], back = row - a.row_run0[row];
  const int C = 2 * a.hk * DK + a.hv * DV;
  const int base = a.conv_w != nullptr ? pos % a.taps : 0;
  const PrepView pv = prep_view<DK, DV, RULE>(a);
  auto input = [&](int ch) {
    const T* x = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.c_off + ch;
    const float xv = ld_elem(x);
    return silu_f32(a.conv_w == nullptr ? xv : conv_channel(a, x, a.stride, xv, back, C, slot, pos, base, ch));
  };
  if (unit < a.hk) {
    float q[DK / 32], k[DK / 32], q2 = 0.f, k2 = 0.f;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
      q[i] = input(unit * DK + 32 * i + lane);
      k[i] = input((a.hk + unit) * DK + 32 * i + lane);
      q2 = fmaf(q[i], q[i], q2); k2 = fmaf(k[i], k[i], k2);
    }
    q2 = warp_sum_f32(q2); k2 = warp_sum_f32(k2);
    const float rq = DELTA ? a.q_scale / sqrtf(q2 + 1e-6f) : 1.f, rk = DELTA ? 1.f / sqrtf(k2 + 1e-6f) : 1.f;
    const size_t o = (static_cast<size_t>(row) * a.hk + unit) * DK + lane;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
      pv.q[o + 32 * i] = q[i] * rq;
      pv.k[o + 32 * i] = k[i] * rk;
    }
    return;
  }
  const int h = unit - a.hk;
  const size_t rh = static_cast<size_t>(row) * a.hv + h;
#pragma unroll
  for (int i = 0; i < DV / 32; ++i) pv.v[rh * DV + 32 * i + lane] = input(2 * a.hk * DK + h * DV + 32 * i + lane);
  if (RULE == kStateSpace && lane == 0) {
    const float dt = softplus_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.b_off + h) + a.dt_bias[h]);
    pv.b[rh] = dt;
    pv.g[rh] = expf(-expf(a.A_log[h]) * dt);
  }
  if (RULE == kScalarDelta && lane == 0) {
    const T* x = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + h;
    pv.b[rh] = sigmoid_f32(ld_elem(x + a.b_off));
    pv.g[rh] = expf(-expf(a.A_log[h]) * softplus_f32(ld_elem(x + a.a_off) + a.dt_bias[h]));
  }
  if (DELTA) {
    const float ea = -expf(a.A_log[h]);
    const float* ar = a.low + static_cast<size_t>(row) * a.low_stride + h * DK + lane;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) pv.g[rh * DK + 32 * i + lane] = expf(ea * softplus_f32(ar[32 * i] + a.dt_bias[h * DK + 32 * i + lane]));
    if (lane == 0) pv.b[rh] = sigmoid_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.b_off + h));
  }
}

// grid (ceil(C / 256), runs)
template <typename T>
__global__ void __launch_bounds__(256) lin_tail_kernel(LinearArgs a, int C) {
  pdl_wait();
  const int ch = blockIdx.x * 256 + threadIdx.x;
  if (ch >= C) return;
  const int first = a.run_start[blockIdx.y], last = a.run_start[blockIdx.y + 1];
  const int slot = a.row_slot[first];
  for (int row = max(first, last - a.taps); row < last; ++row)
    a.ring[(static_cast<size_t>(slot) * a.taps + a.positions[row] % a.taps) * C + ch] =
        ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.c_off + ch);
}

// Block form of the recurrences, 16 tokens at a time.  With gamma_t = g_1 .. g_t (per key channel, products of decays, never a
// quotient) and S the state before the block:
//     delta      W = V - (K * gamma) S,   U = T B W,   T = (I + A)^-1,   A_ts = b_t sum_c k_t k_s (g_(s+1) .. g_t)   (s < t)
//     lightning  U = V
//     O = (Q * gamma) S + P U,            P_ts = sum_c q_t k_s (g_(s+1) .. g_t)                                      (s <= t)
//     S <- gamma_16 * S + (K * g_(t+1) .. g_16)^T U
//     scalar     as delta, with gamma_t a number: gamma_t (K S) instead of (K * gamma) S
//     matrix m.  as state sp. with D = 0, dt_s = w_s
//     state sp.  U = V,  P_ts = (q_t . k_s) (a_(s+1) .. a_t) dt_s + [s = t] D,  O = (a_1 .. a_t) (Q S) + P U,
//                S <- (a_1 .. a_16) S + K^T (dt_s a_(s+1) .. a_16 U)
// lin_block (parallel over blocks and heads) makes K * gamma, Q * gamma, the suffix-weighted keys, gamma_16, T B and P.
// Places behind a run's end hold k = q = v = 0, decay 1 and strength 0: they change nothing.
constexpr int kBlk = 16;

// Sums NV values over PARTS lanes with a halving exchange: every step sends the half of the values the partner keeps.  Lane
// `part` ends with the totals of values [part * n, part * n + n), n = max(NV / PARTS, 1) (NV < PARTS: PARTS / NV lanes share
// value part * NV / PARTS), in v[0 .. n - 1].
template <int NV, int PARTS>
__device__ __forceinline__ void halving_sum(float (&v)[NV], int part) {
  int half = NV / 2;
#pragma unroll
  for (int o = PARTS / 2; o > 0; o >>= 1) {
    if (half >= 1) {
      const bool up = (part & o) != 0;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i) {
        if (i < half) {
          const float give = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
      half >>= 1;
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
  }
}

// The run and the first row of block `blk` (blocks are dealt run by run).
__device__ __forceinline__ bool find_block(const LinearArgs& a, int blk, int& row0, int& n) {
  for (int r = 0; r < a.runs; ++r) {
    const int s = a.run_start[r], len = a.run_start[r + 1] - s, nb = (len + kBlk - 1) / kBlk;
    if (blk < nb) {
      row0 = s + blk * kBlk;
      n = min(kBlk, len - blk * kBlk);
      return true;
    }
    blk -= nb;
  }
  return false;
}

// grid (hv, blocks), 256 threads
template <int DK, int DV, int RULE>
__global__ void __launch_bounds__(256) lin_block_kernel(LinearArgs a) {
  constexpr bool DELTA = RULE == kDelta;
  extern __shared__ __align__(16) float bl_smem[];
  float* ks = bl_smem;                                    // [16][DK]
  float* qs = ks + kBlk * DK;
  float* gs = qs + kBlk * DK;                             // (delta)
  __shared__ float A[kBlk][kBlk + 1], b_s[kBlk];
  pdl_wait();
  const int h = blockIdx.x, blk = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int row0 = 0, n = 0;
  if (!find_block(a, blk, row0, n)) return;
  const int hk = h / (a.hv / a.hk);
  const PrepView pv = prep_view<DK, DV, RULE>(a);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int i = tid; i < kBlk * (DK / 4); i += 256) {
    const int t = i / (DK / 4), c = (i % (DK / 4)) * 4;
    const size_t o = (static_cast<size_t>(row0 + t) * a.hk + hk) * DK + c, og = (static_cast<size_t>(row0 + t) * a.hv + h) * DK + c;
    *reinterpret_cast<float4*>(ks + t * DK + c) = t < n ? *reinterpret_cast<const float4*>(pv.k + o) : zero;
    *reinterpret_cast<float4*>(qs + t * DK + c) = t < n ? *reinterpret_cast<const float4*>(pv.q + o) : zero;
    if (DELTA) *reinterpret_cast<float4*>(gs + t * DK + c) = t < n ? *reinterpret_cast<const float4*>(pv.g + og) : make_float4(1.f, 1.f, 1.f, 1.f);
  }
  if (tid < kBlk) b_s[tid] = DELTA && tid < n ? pv.b[static_cast<size_t>(row0 + tid) * a.hv + h] : 0.f;
  const float dh = DELTA ? 1.f : a.decay[h];
  __syncthreads();
  const size_t bh = static_cast<size_t>(blk) * a.hv + h;
  // ---- products of decays up to and behind every token: two passes over a channel, by different threads where there are enough
  for (int i = tid; i < 2 * DK; i += 256) {
    const int c = i % DK;
    float w = 1.f;
    if (i < DK) {
      for (int t = 0; t < n; ++t) {
        w *= DELTA ? gs[t * DK + c] : dh;
        const size_t o = (static_cast<size_t>(row0 + t) * a.hv + h) * DK + c;
        if (DELTA) pv.kt[o] = ks[t * DK + c] * w;
        pv.qt[o] = qs[t * DK + c] * w;
      }
      pv.gam[bh * DK + c] = w;
    } else {
      for (int t = n - 1; t >= 0; --t) {
        pv.kh[(static_cast<size_t>(row0 + t) * a.hv + h) * DK + c] = ks[t * DK + c] * w;
        w *= DELTA ? gs[t * DK + c] : dh;
      }
    }
  }
  // ---- token pairs: a warp takes the writers s = warp and 15 - warp and walks the readers t >= s
#pragma unroll 1
  for (int which = 0; which < 2; ++which) {
    const int s = which ? kBlk - 1 - warp : warp;
    float run[DK / 32], val[2 * kBlk];
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) run[i] = ks[s * DK + 32 * i + lane];
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
      val[t] = 0.f;
      val[kBlk + t] = 0.f;
      if (t >= s) {
#pragma unroll
        for (int i = 0; i < DK / 32; ++i) {
          const int c = t * DK + 32 * i + lane;
          if (t > s) run[i] *= DELTA ? gs[c] : dh;
          if (DELTA) val[t] = fmaf(run[i], ks[c], val[t]);
          val[kBlk + t] = fmaf(run[i], qs[c], val[kBlk + t]);
        }
      }
    }
    halving_sum<2 * kBlk, 32>(val, lane);
    const int t = lane & (kBlk - 1);
    if (lane < kBlk) A[t][s] = DELTA && t > s ? b_s[t] * val[0] : 0.f;
    else pv.pm[bh * kBlk * kBlk + t * kBlk + s] = t >= s ? val[0] : 0.f;
  }
  if (!DELTA) return;
  __syncthreads();
  // ---- T B: column j of (I + A)^-1 by forward substitution, one lane per column
  if (tid < kBlk) {
    float col[kBlk];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) {
      float acc = i == tid ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) acc = fmaf(-A[i][j], col[j], acc);
      col[i] = acc;
      pv.tb[bh * kBlk * kBlk + i * kBlk + tid] = acc * b_s[tid];
    }
  }
}

// lin_prep of the rules with scalar decays for convolutions of up to four taps: a thread owns four channels of a 16-token block and slides the
// window along in registers.  grid (ceil(C / 512) + 1, blocks), 128 threads; the last column of CTAs makes steps (strengths) and decays.
template <typename T, int DK, int DV, int RULE, int TAPS>
__global__ void __launch_bounds__(128) ssd_prep_kernel(LinearArgs a) {
  pdl_wait();
  int row0 = 0, n = 0;
  if (!find_block(a, blockIdx.y, row0, n)) return;
  const PrepView pv = prep_view<DK, DV, RULE>(a);
  const T* proj = static_cast<const T*>(a.proj) + static_cast<size_t>(row0) * a.stride;
  if (blockIdx.x == gridDim.x - 1) {
    for (int i = threadIdx.x; i < n * a.hv; i += 128) {
      const int t = i / a.hv, h = i % a.hv;
      const float dt = softplus_f32(ld_elem(proj + t * a.stride + (RULE == kScalarDelta ? a.a_off : a.b_off) + h) + a.dt_bias[h]);
      pv.b[static_cast<size_t>(row0) * a.hv + i] = RULE == kScalarDelta ? sigmoid_f32(ld_elem(proj + t * a.stride + a.b_off + h)) : dt;
      pv.g[static_cast<size_t>(row0) * a.hv + i] = expf(-expf(a.A_log[h]) * dt);
    }
    return;
  }
  const int nk = a.hk * DK, C = 2 * nk + a.hv * DV, ch = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (ch >= C) return;
  const int pos = a.positions[row0], back = row0 - a.row_run0[row0];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const T* x = proj + a.c_off + ch;
  const float* ring = a.ring + static_cast<size_t>(a.row_slot[row0]) * TAPS * C + ch;
  float4 w[TAPS], h[TAPS];                                 // h[j]: the input j tokens back
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    w[j] = ld_elem4(a.conv_w + static_cast<size_t>(TAPS - 1 - j) * C + ch);
    h[j] = zero;
    if (j >= 1 && j <= pos) h[j] = j <= back ? ld_elem4(x - j * a.stride) : ld_elem4(ring + static_cast<size_t>((pos - j) % TAPS) * C);
  }
  const float4 bias = a.conv_b != nullptr ? ld_elem4(a.conv_b + ch) : zero;
  float* dst = ch < nk ? pv.q + static_cast<size_t>(row0) * nk + ch
                       : (ch < 2 * nk ? pv.k + static_cast<size_t>(row0) * nk + ch - nk : pv.v + static_cast<size_t>(row0) * a.hv * DV + ch - 2 * nk);
  const int step = ch < 2 * nk ? nk : a.hv * DV;
#pragma unroll 4
  for (int t = 0; t < n; ++t) {
    h[0] = ld_elem4(x + t * a.stride);
    float4 acc = bias;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      acc.x = fmaf(w[j].x, h[j].x, acc.x); acc.y = fmaf(w[j].y, h[j].y, acc.y);
      acc.z = fmaf(w[j].z, h[j].z, acc.z); acc.w = fmaf(w[j].w, h[j].w, acc.w);
    }
    *reinterpret_cast<float4*>(dst + static_cast<size_t>(t) * step) = make_float4(silu_f32(acc.x), silu_f32(acc.y), silu_f32(acc.z), silu_f32(acc.w));
#pragma unroll
    for (int j = TAPS - 1; j > 0; --j) h[j] = h[j - 1];
  }
}

// Matrix memory: q (scaled), k and v as fp32 rows.  grid (ceil(C / 1024), rows), 256 threads.
template <typename T, int DK, int DV>
__global__ void __launch_bounds__(256) matrix_prep_kernel(LinearArgs a) {
  pdl_wait();
  const int nk = a.hk * DK, nv = a.hv * DV, ch = (blockIdx.x * 256 + threadIdx.x) * 4;
  const size_t row = blockIdx.y;
  if (ch >= 2 * nk + nv) return;
  const PrepView pv = prep_view<DK, DV, kMatrix>(a);
  float4 x = ld_elem4(static_cast<const T*>(a.proj) + row * a.stride + a.c_off + ch);
  if (ch < nk) { x.x *= a.q_scale; x.y *= a.q_scale; x.z *= a.q_scale; x.w *= a.q_scale; }
  float* dst = ch < nk ? pv.q + row * nk + ch : (ch < 2 * nk ? pv.k + row * nk + ch - nk : pv.v + row * nv + ch - 2 * nk);
  *reinterpret_cast<float4*>(dst) = x;
}

constexpr int kGateThreads = 512;

// (F, M) of consecutive tokens combine to (F1 + F2, max(M1 + F2, M2)): inclusive scan over the lanes.
__device__ __forceinline__ void gate_scan(float& F, float& M, int lane) {
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
    if (lane >= o) {
      M = fmaxf(Mp + F, M);
      F += Fp;
    }
  }
}

// The running maximum of a run and head, 512 tokens at a time: m_t = max(m + F_t, M_t).  grid (hv, runs)
template <typename T, int DK, int DV>
__global__ void __launch_bounds__(kGateThreads) matrix_gates_kernel(LinearArgs a) {
  constexpr int NW = kGateThreads / 32;
  __shared__ float Fw[NW], Mw[NW], ends[NW + 1];
  pdl_wait();
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int first = a.run_start[blockIdx.y], last = a.run_start[blockIdx.y + 1];
  const PrepView pv = prep_view<DK, DV, kMatrix>(a);
  float* ns = a.nstate + (static_cast<size_t>(a.row_slot[first]) * a.hv + h) * (DK + 4) + DK;
  float m = a.positions[first] == 0 ? 0.f : *ns;
  for (int t0 = first; t0 < last; t0 += kGateThreads) {
    const bool live = t0 + tid < last;
    const float2 g = live ? matrix_gates<T>(a, t0 + tid, h) : make_float2(-INFINITY, 0.f);
    float F = g.y, M = g.x;
    gate_scan(F, M, lane);
    if (lane == 31) { Fw[warp] = F; Mw[warp] = M; }
    __syncthreads();
    if (warp == 0) {                                       // maximum in front of every warp's tokens, and behind all
      float Fs = lane < NW ? Fw[lane] : 0.f, Ms = lane < NW ? Mw[lane] : -INFINITY;
      gate_scan(Fs, Ms, lane);
      if (lane < NW) ends[lane + 1] = fmaxf(m + Fs, Ms);
      if (lane == 0) ends[0] = m;
    }
    __syncthreads();
    const float mw = ends[warp], mt = fmaxf(mw + F, M);
    float before = __shfl_up_sync(0xffffffffu, mt, 1);
    if (lane == 0) before = mw;
    if (live) {
      const size_t o = static_cast<size_t>(t0 + tid) * a.hv + h;
      pv.g[o] = expf(fminf(g.y + before - mt, 0.f));
      pv.b[o] = expf(g.x - mt);
      pv.fl[o] = expf(-mt);
    }
    m = ends[NW];
    __syncthreads();
  }
  if (tid == 0) *ns = m;
}

constexpr int kSsdHeads = 8;

// grid (hk * ceil(heads per group / 8), blocks), 256 threads: thread (t, s) holds q_t . k_s and walks up to 8 heads of the group.
template <int DK, int DV, int RULE>
__global__ void __launch_bounds__(256) ssd_block_kernel(LinearArgs a) {
  __shared__ float ks[kBlk][DK + 1], qs[kBlk][DK + 1];
  __shared__ float as[kSsdHeads][kBlk], ds[kSsdHeads][kBlk];
  pdl_wait();
  const int ratio = a.hv / a.hk, chunks = (ratio + kSsdHeads - 1) / kSsdHeads;
  const int hk = blockIdx.x / chunks, h0 = hk * ratio + (blockIdx.x % chunks) * kSsdHeads;
  const int nh = min(kSsdHeads, (hk + 1) * ratio - h0), blk = blockIdx.y, tid = threadIdx.x;
  int row0 = 0, n = 0;
  if (!find_block(a, blk, row0, n)) return;
  const PrepView pv = prep_view<DK, DV, RULE>(a);
  for (int i = tid; i < kBlk * DK; i += 256) {
    const int t = i / DK, c = i % DK;
    const size_t o = (static_cast<size_t>(row0 + t) * a.hk + hk) * DK + c;
    ks[t][c] = t < n ? pv.k[o] : 0.f;
    qs[t][c] = t < n ? pv.q[o] : 0.f;
  }
  for (int i = tid; i < nh * kBlk; i += 256) {
    const int h = i / kBlk, t = i % kBlk;
    const size_t o = static_cast<size_t>(row0 + t) * a.hv + h0 + h;
    as[h][t] = t < n ? pv.g[o] : 1.f;
    ds[h][t] = t < n ? pv.b[o] : 0.f;
  }
  __syncthreads();
  const int t = tid / kBlk, s = tid % kBlk;
  float dot = 0.f;
  if (s <= t) {
#pragma unroll 8
    for (int c = 0; c < DK; ++c) dot = fmaf(qs[t][c], ks[s][c], dot);
  }
  for (int h = 0; h < nh; ++h) {
    const size_t bh = static_cast<size_t>(blk) * a.hv + h0 + h;
    float p = 0.f;
    if (s <= t) {
      p = dot;
      for (int j = s + 1; j <= t; ++j) p *= as[h][j];
      p *= ds[h][s];
      if (RULE == kStateSpace && s == t && t < n) p += a.skip[h0 + h];
    }
    pv.pm[bh * kBlk * kBlk + tid] = p;
    if (tid < 2 * kBlk) {
      float w = 1.f;
      if (tid < kBlk) {
        for (int j = 0; j <= tid; ++j) w *= as[h][j];
      } else {
        for (int j = kBlk - 1; j > tid - kBlk; --j) w *= as[h][j];
        w *= ds[h][tid - kBlk];
      }
      pv.gam[bh * 2 * kBlk + tid] = w;
    }
  }
}

// The same for the scalar delta rule: thread (t, s) holds q_t . k_s and k_t . k_s of the raw vectors, whose lengths become factors;
// (I + A)^-1 of up to 8 heads side by side, one lane per column.
template <int DK, int DV>
__global__ void __launch_bounds__(256) gated_block_kernel(LinearArgs a) {
  __shared__ float ks[kBlk][DK + 1], qs[kBlk][DK + 1];
  __shared__ float as[kSsdHeads][kBlk], bs[kSsdHeads][kBlk], rq[kBlk], rk[kBlk];
  __shared__ float A[kSsdHeads][kBlk][kBlk + 1];
  pdl_wait();
  const int ratio = a.hv / a.hk, chunks = (ratio + kSsdHeads - 1) / kSsdHeads;
  const int hk = blockIdx.x / chunks, h0 = hk * ratio + (blockIdx.x % chunks) * kSsdHeads;
  const int nh = min(kSsdHeads, (hk + 1) * ratio - h0), blk = blockIdx.y, tid = threadIdx.x;
  int row0 = 0, n = 0;
  if (!find_block(a, blk, row0, n)) return;
  const PrepView pv = prep_view<DK, DV, kScalarDelta>(a);
  for (int i = tid; i < kBlk * DK; i += 256) {
    const int t = i / DK, c = i % DK;
    const size_t o = (static_cast<size_t>(row0 + t) * a.hk + hk) * DK + c;
    ks[t][c] = t < n ? pv.k[o] : 0.f;
    qs[t][c] = t < n ? pv.q[o] : 0.f;
  }
  for (int i = tid; i < nh * kBlk; i += 256) {
    const int h = i / kBlk, t = i % kBlk;
    const size_t o = static_cast<size_t>(row0 + t) * a.hv + h0 + h;
    as[h][t] = t < n ? pv.g[o] : 1.f;
    bs[h][t] = t < n ? pv.b[o] : 0.f;
  }
  __syncthreads();
  for (int t = tid / 32; t < kBlk; t += 8) {
    float q2 = 0.f, k2 = 0.f;
    for (int c = tid & 31; c < DK; c += 32) {
      q2 = fmaf(qs[t][c], qs[t][c], q2);
      k2 = fmaf(ks[t][c], ks[t][c], k2);
    }
    q2 = warp_sum_f32(q2); k2 = warp_sum_f32(k2);
    if ((tid & 31) == 0) { rq[t] = a.q_scale / sqrtf(q2 + 1e-6f); rk[t] = 1.f / sqrtf(k2 + 1e-6f); }
  }
  const int t = tid / kBlk, s = tid % kBlk;
  float dq = 0.f, dk = 0.f;
  if (s <= t) {
#pragma unroll 8
    for (int c = 0; c < DK; ++c) {
      dq = fmaf(qs[t][c], ks[s][c], dq);
      dk = fmaf(ks[t][c], ks[s][c], dk);
    }
  }
  __syncthreads();
  dq *= rq[t] * rk[s];
  dk *= rk[t] * rk[s];
  for (int h = 0; h < nh; ++h) {
    const size_t bh = static_cast<size_t>(blk) * a.hv + h0 + h;
    float w = 1.f;
    if (s <= t)
      for (int j = s + 1; j <= t; ++j) w *= as[h][j];
    pv.pm[bh * kBlk * kBlk + tid] = s <= t ? dq * w : 0.f;
    A[h][t][s] = s < t ? bs[h][t] * dk * w : 0.f;
    if (tid < 4 * kBlk) {                                  // factors of Q S, of the writes, of K S; gamma_16
      const int i = tid % kBlk, what = tid / kBlk;
      float f = 1.f;
      if (what == 1) {
        for (int j = kBlk - 1; j > i; --j) f *= as[h][j];
        f *= rk[i];
      } else {
        for (int j = 0; j <= (what == 3 ? kBlk - 1 : i); ++j) f *= as[h][j];
        f *= what == 0 ? rq[i] : (what == 2 ? rk[i] : 1.f);
      }
      pv.gam[bh * 4 * kBlk + tid] = f;
    }
  }
  __syncthreads();
  if (tid < nh * kBlk) {
    const int h = tid / kBlk, c = tid % kBlk;
    float* tb = pv.tb + (static_cast<size_t>(blk) * a.hv + h0 + h) * kBlk * kBlk;
    float col[kBlk];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) {
      float acc = i == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) acc = fmaf(-A[h][i][j], col[j], acc);
      col[i] = acc;
      tb[i * kBlk + c] = acc * bs[h][c];
    }
  }
}

constexpr int kScanCols = 32;

template <int DK, int RULE>
struct ScanGeom {
  static constexpr int kParts = DK >= 128 ? 32 : DK / 4;    // threads that share a column
  static constexpr int kThreads = kParts * (kScanCols / 4) + (RULE == kMatrix ? 32 : 0);
  static constexpr int kNI = DK / (4 * kParts);
  // floats of one staging buffer
  static constexpr int kQ = 0, kH = kBlk * DK, kK = 2 * kBlk * DK;
  static constexpr int kV = kK + (RULE == kDelta ? kBlk * DK : 0);
  static constexpr int kP = kV + kBlk * kScanCols, kT = kP + kBlk * kBlk;
  static constexpr int kG = kT + (is_delta(RULE) ? kBlk * kBlk : 0);
  static constexpr int kGam = RULE == kStateSpace || RULE == kMatrix ? 2 * kBlk : (RULE == kScalarDelta ? 4 * kBlk : DK);   // factors of a block and head
  static constexpr int kTotal = kG + kGam;
};

// Block-sequential pass.  A CTA owns 32 columns of one head's state in registers: a thread 4 columns and the rows
// 4 part + 4 PARTS i + e; the PARTS lanes of a column group sit in one warp, so a group works through a block on its own and
// the CTA only meets at the staging buffers (the next block streams in with cp.async meanwhile).
// Matrix memory: the last warp's first group holds n (in the first CTA of a head).  grid (DV / 32, hv, runs)
template <int DK, int DV, int RULE>
__global__ void __launch_bounds__(ScanGeom<DK, RULE>::kThreads) lin_scan_kernel(LinearArgs a) {
  constexpr bool DELTA = is_delta(RULE), CH = RULE == kDelta, SCALAR = scalar_decay(RULE);
  using G = ScanGeom<DK, RULE>;
  constexpr int NI = G::kNI, PARTS = G::kParts, NT = G::kThreads;
  constexpr int NV = 4 * kBlk, CNT = NV / PARTS;            // values of a group's block; totals per lane (2, 4 or 8)
  extern __shared__ __align__(16) float sc_smem[];          // [2][G::kTotal], then W and U of every group [8][2][64]
  pdl_wait();
  const int tid = threadIdx.x, cg = tid / PARTS, part = tid % PARTS;
  const int h = blockIdx.y, jb = blockIdx.x * kScanCols, j0 = jb + 4 * cg;
  const int first = a.run_start[blockIdx.z], last = a.run_start[blockIdx.z + 1];
  int blk = 0;
  for (int r = 0; r < static_cast<int>(blockIdx.z); ++r) blk += (a.run_start[r + 1] - a.run_start[r] + kBlk - 1) / kBlk;
  const int slot = a.row_slot[first], hk = SCALAR ? h / (a.hv / a.hk) : 0;
  const PrepView pv = prep_view<DK, DV, RULE>(a);
  float* ws = sc_smem + 2 * G::kTotal + cg * 2 * NV;        // [16][4] W
  float* us = ws + NV;                                      // [16][4] U
  float* sp = a.state + (static_cast<size_t>(slot) * a.hv + h) * DK * DV + j0;
  const bool fresh = a.positions[first] == 0;
  const bool ones = RULE == kMatrix && cg >= kScanCols / 4;  // the warp for n: column 0 of its first group
  float* ns = ones ? a.nstate + (static_cast<size_t>(slot) * a.hv + h) * (DK + 4) : nullptr;
  float s[NI][4][4];                                        // [i][row e][column]
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (ones) {
        s[i][e][0] = cg == kScanCols / 4 && !fresh ? ns[4 * PARTS * i + 4 * part + e] : 0.f;
        s[i][e][1] = s[i][e][2] = s[i][e][3] = 0.f;
        continue;
      }
      const float4 v = fresh ? make_float4(0.f, 0.f, 0.f, 0.f)
                             : *reinterpret_cast<const float4*>(sp + static_cast<size_t>(4 * PARTS * i + 4 * part + e) * DV);
      s[i][e][0] = v.x; s[i][e][1] = v.y; s[i][e][2] = v.z; s[i][e][3] = v.w;
    }
  auto stage = [&](int buf, int t0, int b) {
    float* d = sc_smem + buf * G::kTotal;
    const int n = min(kBlk, last - t0);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = tid; i < kBlk * (DK / 4); i += NT) {
      const int t = i / (DK / 4), c = (i % (DK / 4)) * 4;
      const size_t o = SCALAR ? (static_cast<size_t>(t0 + t) * a.hk + hk) * DK + c : (static_cast<size_t>(t0 + t) * a.hv + h) * DK + c;
      if (t < n) {
        cp_async_16(d + G::kQ + t * DK + c, (SCALAR ? pv.q : pv.qt) + o);
        cp_async_16(d + G::kH + t * DK + c, (SCALAR ? pv.k : pv.kh) + o);
        if (CH) cp_async_16(d + G::kK + t * DK + c, pv.kt + o);
      } else {
        *reinterpret_cast<float4*>(d + G::kQ + t * DK + c) = zero;
        *reinterpret_cast<float4*>(d + G::kH + t * DK + c) = zero;
        if (CH) *reinterpret_cast<float4*>(d + G::kK + t * DK + c) = zero;
      }
    }
    for (int i = tid; i < kBlk * (kScanCols / 4); i += NT) {
      const int t = i / (kScanCols / 4), c = (i % (kScanCols / 4)) * 4;
      if (t < n) cp_async_16(d + G::kV + t * kScanCols + c, pv.v + (static_cast<size_t>(t0 + t) * a.hv + h) * DV + jb + c);
      else *reinterpret_cast<float4*>(d + G::kV + t * kScanCols + c) = zero;
    }
    const size_t bh = static_cast<size_t>(b) * a.hv + h;
    for (int i = tid * 4; i < kBlk * kBlk; i += NT * 4) {
      cp_async_16(d + G::kP + i, pv.pm + bh * kBlk * kBlk + i);
      if (DELTA) cp_async_16(d + G::kT + i, pv.tb + bh * kBlk * kBlk + i);
    }
    for (int i = tid * 4; i < G::kGam; i += NT * 4) cp_async_16(d + G::kG + i, pv.gam + bh * G::kGam + i);
    cp_async_group_commit();
  };
  // partial products of 16 staged rows with this thread's part of the state, summed over the group
  auto rows_times_state = [&](const float* m, float (&val)[NV]) {
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
#pragma unroll
      for (int c = 0; c < 4; ++c) val[4 * t + c] = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 m4 = *reinterpret_cast<const float4*>(m + t * DK + 4 * PARTS * i + 4 * part);
        const float mf[4] = {m4.x, m4.y, m4.z, m4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < 4; ++c) val[4 * t + c] = fmaf(mf[e], s[i][e][c], val[4 * t + c]);
      }
    }
    halving_sum<NV, PARTS>(val, part);
  };
  // rows of a 16 x 16 matrix (row-major) times a group's [16][4] block `x` (row stride xs): this lane's CNT entries
  auto pairs_times = [&](const float* m, const float* x, int xs, float (&out)[CNT]) {
#pragma unroll
    for (int i = 0; i < CNT; ++i) {
      const int t = (part * CNT + i) / 4, c = (part * CNT + i) % 4;
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < kBlk; j += 4) {
        const float4 m4 = *reinterpret_cast<const float4*>(m + t * kBlk + j);
        acc = fmaf(m4.x, x[j * xs + c], acc);
        acc = fmaf(m4.y, x[(j + 1) * xs + c], acc);
        acc = fmaf(m4.z, x[(j + 2) * xs + c], acc);
        acc = fmaf(m4.w, x[(j + 3) * xs + c], acc);
      }
      out[i] = acc;
    }
  };
  float* one_v = sc_smem + 2 * G::kTotal;                   // matrix memory: [16] rows of 32 columns, ones in the first (no W and U there)
  if (RULE == kMatrix)
    for (int i = tid; i < kBlk * kScanCols; i += NT) one_v[i] = i % kScanCols == 0 ? 1.f : 0.f;
  stage(0, first, blk);
  int buf = 0;
  for (int t0 = first; t0 < last; t0 += kBlk, buf ^= 1, ++blk) {
    if (t0 + kBlk < last) {
      stage(buf ^ 1, t0 + kBlk, blk + 1);
      cp_async_group_wait<1>();
    } else {
      cp_async_group_wait<0>();
    }
    __syncthreads();
    const float* d = sc_smem + buf * G::kTotal;
    const float* vb = ones ? one_v : d + G::kV + 4 * cg;                   // [16] rows of 32 columns, this group's 4
    const int n = min(kBlk, last - t0);
    if (ones && blockIdx.x > 0) {                           // n has its place in the first CTA
      __syncthreads();
      continue;
    }
    float val[NV], x[CNT];
    if (DELTA) {
      rows_times_state(d + (CH ? G::kK : G::kH), val);
#pragma unroll
      for (int i = 0; i < CNT; ++i) {
        const int idx = part * CNT + i;
        ws[idx] = fmaf(CH ? -1.f : -d[G::kG + 2 * kBlk + idx / 4], val[i], vb[(idx / 4) * kScanCols + idx % 4]);
      }
      __syncwarp();
      pairs_times(d + G::kT, ws, 4, x);
#pragma unroll
      for (int i = 0; i < CNT; ++i) us[part * CNT + i] = x[i];
    }
    rows_times_state(d + G::kQ, val);
    __syncwarp();
    const float* u = DELTA ? us : vb;
    constexpr int ustride = DELTA ? 4 : kScanCols;
    pairs_times(d + G::kP, u, ustride, x);
#pragma unroll
    for (int i = 0; i < CNT; ++i) {
      const int idx = part * CNT + i;
      const float w = SCALAR ? d[G::kG + idx / 4] : 1.f;
      if (ones) {
        const size_t rh = static_cast<size_t>(t0 + idx / 4) * a.hv + h;
        if (idx / 4 < n && cg == kScanCols / 4 && idx % 4 == 0) a.den[rh] = matrix_den(fmaf(w, val[i], x[i]), pv.fl[rh]);
      } else if (idx / 4 < n && j0 + idx % 4 < a.ow) a.o[(static_cast<size_t>(t0 + idx / 4) * a.hv + h) * a.ow + j0 + idx % 4] = fmaf(w, val[i], x[i]);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      float4 g4;
      if (SCALAR) g4.x = g4.y = g4.z = g4.w = d[G::kG + (DELTA ? 3 * kBlk : kBlk - 1)];
      else g4 = *reinterpret_cast<const float4*>(d + G::kG + 4 * PARTS * i + 4 * part);
      const float gf[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[i][e][c] *= gf[e];
    }
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
      const float4 u4 = *reinterpret_cast<const float4*>(u + t * ustride);
      const float w = SCALAR ? d[G::kG + kBlk + t] : 1.f;
      const float uf[4] = {u4.x * w, u4.y * w, u4.z * w, u4.w * w};
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(d + G::kH + t * DK + 4 * PARTS * i + 4 * part);
        const float kf[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < 4; ++c) s[i][e][c] = fmaf(kf[e], uf[c], s[i][e][c]);
      }
    }
    __syncthreads();                                        // this buffer's readers are done before it is staged again
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (ones) {
        if (cg == kScanCols / 4 && blockIdx.x == 0) ns[4 * PARTS * i + 4 * part + e] = s[i][e][0];
      } else {
        *reinterpret_cast<float4*>(sp + static_cast<size_t>(4 * PARTS * i + 4 * part + e) * DV) =
            make_float4(s[i][e][0], s[i][e][1], s[i][e][2], s[i][e][3]);
      }
    }
}

template <typename T, int DK, int DV, int RULE>
static int launch_lin(const LinearArgs& a, int decode, cudaStream_t st) {
  constexpr bool DELTA = is_delta(RULE);
  using G = LinGeom<DK, DV>;
  if (decode) {
    const size_t smem = static_cast<size_t>(G::kParts) * DV * sizeof(float) * (DELTA ? 2 : 1);
    static_assert(static_cast<size_t>(G::kParts) * DV * 8 <= 48 * 1024, "decode reduction buffer");
    lin_decode_kernel<T, DK, DV, RULE><<<dim3(a.hv, a.rows), G::kThreads, smem, st>>>(a);
    DGPP_CUDA_OK(cudaGetLastError());
    return 0;
  }
  constexpr size_t smem = (2 * ScanGeom<DK, RULE>::kTotal + 8 * 2 * 4 * kBlk) * sizeof(float);
  constexpr size_t bsmem = (DELTA ? 3 : 2) * static_cast<size_t>(kBlk) * DK * sizeof(float);
  static bool attr = false;
  if (!attr) {
    if constexpr (!scalar_decay(RULE))
      DGPP_CUDA_OK(cudaFuncSetAttribute(lin_block_kernel<DK, DV, RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bsmem)));
    DGPP_CUDA_OK(cudaFuncSetAttribute(lin_scan_kernel<DK, DV, RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    attr = true;
  }
  bool prepared = false;
  if constexpr (RULE == kMatrix) {
    matrix_prep_kernel<T, DK, DV><<<dim3(dgpp_ceil_div(2 * a.hk * DK + a.hv * DV, 1024), a.rows), 256, 0, st>>>(a);
    DGPP_CUDA_OK(cudaGetLastError());
    matrix_gates_kernel<T, DK, DV><<<dim3(a.hv, a.runs), kGateThreads, 0, st>>>(a);
    prepared = true;
  } else if constexpr (scalar_decay(RULE)) {
    const dim3 grid(dgpp_ceil_div(2 * a.hk * DK + a.hv * DV, 512) + 1, a.blocks);
    prepared = a.taps <= 4 && a.stride % 4 == 0 && a.c_off % 4 == 0;
    if (!prepared) {}
    else if (a.taps == 1) ssd_prep_kernel<T, DK, DV, RULE, 1><<<grid, 128, 0, st>>>(a);
    else if (a.taps == 2) ssd_prep_kernel<T, DK, DV, RULE, 2><<<grid, 128, 0, st>>>(a);
    else if (a.taps == 3) ssd_prep_kernel<T, DK, DV, RULE, 3><<<grid, 128, 0, st>>>(a);
    else ssd_prep_kernel<T, DK, DV, RULE, 4><<<grid, 128, 0, st>>>(a);
  }
  if constexpr (RULE != kMatrix)
    if (!prepared) lin_prep_kernel<T, DK, DV, RULE><<<dgpp_ceil_div(a.rows * (a.hk + a.hv), 8), 256, 0, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  const dim3 groups(a.hk * dgpp_ceil_div(a.hv / a.hk, kSsdHeads), a.blocks);
  if constexpr (RULE == kStateSpace || RULE == kMatrix) ssd_block_kernel<DK, DV, RULE><<<groups, 256, 0, st>>>(a);
  else if constexpr (RULE == kScalarDelta) gated_block_kernel<DK, DV><<<groups, 256, 0, st>>>(a);
  else lin_block_kernel<DK, DV, RULE><<<dim3(a.hv, a.blocks), 256, bsmem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  lin_scan_kernel<DK, DV, RULE><<<dim3(DV / kScanCols, a.hv, a.runs), ScanGeom<DK, RULE>::kThreads, smem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  if (a.conv_w != nullptr) {
    const int C = 2 * a.hk * DK + a.hv * DV;
    lin_tail_kernel<T><<<dim3(dgpp_ceil_div(C, 256), a.runs), 256, 0, st>>>(a, C);
    DGPP_CUDA_OK(cudaGetLastError());
  }
  return 0;
}

template <typename T, int RULE>
static int launch_lin_dims(const LinearArgs& a, int DK, int DV, int decode, cudaStream_t st) {
#define DGPP_LIN_CASE(K, V) if (DK == K && DV == V) return launch_lin<T, K, V, RULE>(a, decode, st);
  DGPP_LIN_CASE(32, 32) DGPP_LIN_CASE(32, 64) DGPP_LIN_CASE(32, 128) DGPP_LIN_CASE(32, 256)
  DGPP_LIN_CASE(64, 32) DGPP_LIN_CASE(64, 64) DGPP_LIN_CASE(64, 128) DGPP_LIN_CASE(64, 256)
  DGPP_LIN_CASE(128, 32) DGPP_LIN_CASE(128, 64) DGPP_LIN_CASE(128, 128) DGPP_LIN_CASE(128, 256)
  DGPP_LIN_CASE(256, 32) DGPP_LIN_CASE(256, 64) DGPP_LIN_CASE(256, 128) DGPP_LIN_CASE(256, 256)
#undef DGPP_LIN_CASE
  dgpp_set_error("linear_state: head widths %d x %d (padded to 32, 64, 128 or 256)", DK, DV);
  return -1;
}


// The arguments that every rule has; entry points add their own.
static inline LinearArgs lin_args(const void* proj, int64_t stride, int c_off, int b_off, const void* conv_w, void* ring, int taps,
                                  const void* A_log, const void* dt_bias, void* state, const void* row_slot, const void* positions,
                                  const void* run_start, const void* row_run0, void* prep, void* o, int rows, int runs, int blocks, int hk,
                                  int hv, int vdim, int ow) {
  LinearArgs a;
  memset(&a, 0, sizeof(a));
  a.proj = proj; a.stride = stride; a.c_off = c_off; a.b_off = b_off;
  a.conv_w = static_cast<const float*>(conv_w); a.ring = static_cast<float*>(ring); a.taps = taps;
  a.A_log = static_cast<const float*>(A_log); a.dt_bias = static_cast<const float*>(dt_bias);
  a.state = static_cast<float*>(state);
  a.row_slot = static_cast<const int32_t*>(row_slot); a.positions = static_cast<const int32_t*>(positions);
  a.run_start = static_cast<const int32_t*>(run_start); a.row_run0 = static_cast<const int32_t*>(row_run0);
  a.prep = static_cast<float*>(prep); a.o = static_cast<float*>(o);
  a.rows = rows; a.runs = runs; a.blocks = blocks; a.hk = hk; a.hv = hv; a.vdim = vdim; a.ow = ow;
  return a;
}

static inline int lin_check(const LinearArgs& a, int DV, int decode) {
  DGPP_REQUIRE(a.hk > 0 && a.hv % a.hk == 0, "linear_state: %d value heads over %d key heads", a.hv, a.hk);
  DGPP_REQUIRE(a.vdim >= 1 && a.vdim <= DV, "linear_state: %d true columns of %d", a.vdim, DV);
  DGPP_REQUIRE(decode || (a.blocks >= 1 && a.blocks <= 65535), "linear_state: %d blocks", a.blocks);
  DGPP_REQUIRE(a.rows >= 0 && a.rows <= 65535 && a.runs <= 65535, "linear_state: %d rows in %d runs", a.rows, a.runs);
  DGPP_REQUIRE(a.conv_w == nullptr || (a.taps >= 1 && a.ring), "linear_state: a convolution of %d taps needs its ring", a.taps);
  DGPP_REQUIRE(decode || (a.run_start && a.row_run0 && a.prep && a.o), "linear_state: runs need their bounds and scratch");
  return 0;
}

}  // namespace dgpp

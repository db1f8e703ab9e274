// Linear-attention layers whose memory is one fp32 matrix S [DK, DV] per head and request:
//
//   channel delta rule   S <- g_t * S (a decay per key channel);  u = b_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
//                        q, k, v pass a causal depthwise convolution and silu, q and k become unit vectors, q is scaled;
//                        g_t = exp(-exp(A) softplus(a_t + dt)),  b_t = sigmoid(beta_t)
//   lightning            S <- d_h * S + k_t v_t^T (a constant decay per head);  o_t = S^T q_t;  q, k, v = silu(projection)
//
// Both are one kernel family (template flag DELTA).  A pass carries runs of consecutive tokens of any number of requests:
// run r = rows [run_start[r], run_start[r + 1]) of the request in state slot row_slot[first row].
//
//   lin_decode   runs of one token: convolution, norms, gates, state update and read-out of a (row, head) in one CTA with
//                the whole S in registers; the delta rule's output norm and gate are fused in as well
//   lin_prep     token-parallel part of longer runs -> fp32 scratch (unit q / k, their dot product, v, decays, strengths)
//   lin_scan     token-sequential part: one CTA per (32 state columns, head, run), S in registers, the next tokens' operands
//                streaming in with cp.async while the current ones are consumed
//   lin_tail     the newest inputs of the convolution go to the request's ring after every reader is done
//
// o_t is taken as (g S)^T q + (k . q) u, the read-out after the write, so both reductions over the key channels run
// together.  A request's first token (position 0) starts from S = 0 and from zeros before it: a slot needs no clearing
// between requests.  The convolution's history is a ring of `taps` inputs per channel, entry p % taps for position p: a
// token never overwrites an entry that its own window reads, so decode CTAs of heads that share key heads do not race.
#include <math.h>
#include <string.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

struct LinearArgs {
  const void* proj;         // [rows, stride] (T): conv channels q (hk * DK) | k (hk * DK) | v (hv * DV) from column c_off
  int64_t stride;
  int c_off, b_off;         // b_off: raw write strengths [hv] (delta)
  const float* low;         // [rows, low_stride] fp32: raw decays [hv * DK], then raw output gates [hv * DV] (delta)
  int64_t low_stride;
  const float* conv_w;      // [taps, C] (last row: the current token); null: no convolution
  float* ring;              // [slots, taps, C]
  const float* A_log;       // [hv]
  const float* dt_bias;     // [hv * DK]
  const float* decay;       // [hv] (lightning)
  float* state;             // [slots, hv, DK, DV]
  const int32_t* row_slot;  // [rows]
  const int32_t* positions; // [rows]
  const int32_t* run_start; // [runs + 1]
  const int32_t* row_run0;  // [rows] first row of the row's run
  float* prep;              // scratch (see lin_prep)
  float* o;                 // [rows, hv * DV] fp32 read-outs (scan; lightning decode)
  void* out;                // [rows, out_stride] (T): normed and gated read-outs (delta decode)
  int64_t out_stride;
  const float* norm_w;      // [DV]
  int rows, runs, hk, hv, taps, vdim;
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
  float acc = a.conv_w[static_cast<size_t>(a.taps - 1) * C + ch] * xv;
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

__device__ __forceinline__ float4 fma4(float4 s, float a, float4 acc) {
  acc.x = fmaf(s.x, a, acc.x); acc.y = fmaf(s.y, a, acc.y); acc.z = fmaf(s.z, a, acc.z); acc.w = fmaf(s.w, a, acc.w);
  return acc;
}

// grid (hv, rows)
template <typename T, int DK, int DV, bool DELTA>
__global__ void __launch_bounds__(LinGeom<DK, DV>::kThreads) lin_decode_kernel(LinearArgs a) {
  using G = LinGeom<DK, DV>;
  constexpr int NT = G::kThreads, PER = G::kPer, PARTS = G::kParts;
  extern __shared__ __align__(16) float ld_smem[];
  float* red_n = ld_smem;                                 // [PARTS][DV]
  float* red_m = red_n + PARTS * DV;                      // [PARTS][DV] (delta)
  __shared__ float qs[DK], ks[DK], gs[DK];
  __shared__ __align__(16) float vs[DV], us[DV];
  __shared__ float scal[3];                               // |q|^2, |k|^2, q . k
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
    acc = silu_f32(acc);
    if (c < DK) qs[c] = acc;
    else if (c < 2 * DK) ks[c - DK] = acc;
    else vs[c - 2 * DK] = acc;
  }
  float beta = 1.f;
  if (DELTA) {
    const float ea = -expf(a.A_log[h]);
    const float* ar = a.low + static_cast<size_t>(row) * a.low_stride + h * DK;
    for (int c = tid; c < DK; c += NT) gs[c] = expf(ea * softplus_f32(ar[c] + a.dt_bias[h * DK + c]));
    beta = sigmoid_f32(ld_elem(static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.b_off + h));
  }
  __syncthreads();
  if (tid < 32) {
    float q2 = 0.f, k2 = 0.f, qk = 0.f;
    for (int c = tid; c < DK; c += 32) {
      q2 = fmaf(qs[c], qs[c], q2);
      k2 = fmaf(ks[c], ks[c], k2);
      qk = fmaf(qs[c], ks[c], qk);
    }
    q2 = warp_sum_f32(q2); k2 = warp_sum_f32(k2); qk = warp_sum_f32(qk);
    if (tid == 0) { scal[0] = q2; scal[1] = k2; scal[2] = qk; }
  }
  // ---- decay, both reductions
  const float dh = DELTA ? 1.f : a.decay[h];
  float4 n4 = make_float4(0.f, 0.f, 0.f, 0.f), m4 = n4;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int r = part + PARTS * i;
    const float g = DELTA ? gs[r] : dh;
    s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
    n4 = fma4(s[i], qs[r], n4);
    if (DELTA) m4 = fma4(s[i], ks[r], m4);
  }
  *reinterpret_cast<float4*>(red_n + part * DV + 4 * cg) = n4;
  if (DELTA) *reinterpret_cast<float4*>(red_m + part * DV + 4 * cg) = m4;
  __syncthreads();
  const float rq = DELTA ? a.q_scale / sqrtf(scal[0] + 1e-6f) : 1.f, rk = DELTA ? 1.f / sqrtf(scal[1] + 1e-6f) : 1.f;
  const float qk = scal[2] * rq * rk;
  float ss = 0.f;
  for (int c = tid; c < DV; c += NT) {
    float n = 0.f, m = 0.f;
#pragma unroll
    for (int w = 0; w < PARTS; ++w) {
      n += red_n[w * DV + c];
      if (DELTA) m += red_m[w * DV + c];
    }
    const float u = DELTA ? beta * (vs[c] - m * rk) : vs[c];
    const float o = n * rq + qk * u;
    us[c] = u * rk;                              // the key's norm rides on u
    ss = fmaf(o, o, ss);
    if (DELTA) vs[c] = o;
    else a.o[(static_cast<size_t>(row) * a.hv + h) * DV + c] = o;
  }
  __syncthreads();
  const float4 u4 = *reinterpret_cast<const float4*>(us + 4 * cg);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int r = part + PARTS * i;
    sp[static_cast<size_t>(r) * G::kCols4] = fma4(u4, ks[r], s[i]);
  }
  if (DELTA) {
    const float r = 1.f / sqrtf(block_sum_f32(ss, scratch) / static_cast<float>(a.vdim) + a.eps);
    const float* gt = a.low + static_cast<size_t>(row) * a.low_stride + a.hv * DK + h * DV;
    T* dst = static_cast<T*>(a.out) + static_cast<size_t>(row) * a.out_stride + h * DV;
    for (int c = tid; c < DV; c += NT) st_elem(dst + c, vs[c] * r * a.norm_w[c] * sigmoid_f32(gt[c]));
  }
}

// Scratch layout of lin_prep (fp32): q [rows, hk, DK] | k [rows, hk, DK] | v [rows, hv, DV] | decay [rows, hv, DK] (delta)
// | q . k [rows, hk] | strength [rows, hv] (delta)
struct PrepView {
  float *q, *k, *v, *g, *qk, *b;
};
template <int DK, int DV, bool DELTA>
__device__ __forceinline__ PrepView prep_view(const LinearArgs& a) {
  PrepView p;
  const size_t R = a.rows;
  p.q = a.prep;
  p.k = p.q + R * a.hk * DK;
  p.v = p.k + R * a.hk * DK;
  p.g = p.v + R * a.hv * DV;
  p.qk = p.g + (DELTA ? R * a.hv * DK : 0);
  p.b = p.qk + R * a.hk;
  return p;
}

// One warp per (row, unit): units < hk prepare a key head, the others a value head.
template <typename T, int DK, int DV, bool DELTA>
__global__ void __launch_bounds__(256) lin_prep_kernel(LinearArgs a) {
  pdl_wait();
  const int lane = threadIdx.x & 31, units = a.hk + a.hv;
  const int warp = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (warp >= a.rows * units) return;
  const int row = warp / units, unit = warp % units;
  const int slot = a.row_slot[row], pos = a.positions[row], back = row - a.row_run0[row];
  const int C = 2 * a.hk * DK + a.hv * DV;
  const int base = a.conv_w != nullptr ? pos % a.taps : 0;
  const PrepView pv = prep_view<DK, DV, DELTA>(a);
  auto input = [&](int ch) {
    const T* x = static_cast<const T*>(a.proj) + static_cast<size_t>(row) * a.stride + a.c_off + ch;
    const float xv = ld_elem(x);
    return silu_f32(a.conv_w == nullptr ? xv : conv_channel(a, x, a.stride, xv, back, C, slot, pos, base, ch));
  };
  if (unit < a.hk) {
    float q[DK / 32], k[DK / 32], q2 = 0.f, k2 = 0.f, qk = 0.f;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
      q[i] = input(unit * DK + 32 * i + lane);
      k[i] = input((a.hk + unit) * DK + 32 * i + lane);
      q2 = fmaf(q[i], q[i], q2); k2 = fmaf(k[i], k[i], k2); qk = fmaf(q[i], k[i], qk);
    }
    q2 = warp_sum_f32(q2); k2 = warp_sum_f32(k2); qk = warp_sum_f32(qk);
    const float rq = DELTA ? a.q_scale / sqrtf(q2 + 1e-6f) : 1.f, rk = DELTA ? 1.f / sqrtf(k2 + 1e-6f) : 1.f;
    const size_t o = (static_cast<size_t>(row) * a.hk + unit) * DK + lane;
#pragma unroll
    for (int i = 0; i < DK / 32; ++i) {
      pv.q[o + 32 * i] = q[i] * rq;
      pv.k[o + 32 * i] = k[i] * rk;
    }
    if (lane == 0) pv.qk[static_cast<size_t>(row) * a.hk + unit] = qk * rq * rk;
    return;
  }
  const int h = unit - a.hk;
  const size_t rh = static_cast<size_t>(row) * a.hv + h;
#pragma unroll
  for (int i = 0; i < DV / 32; ++i) pv.v[rh * DV + 32 * i + lane] = input(2 * a.hk * DK + h * DV + 32 * i + lane);
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

// Token-sequential pass.  A CTA owns 32 columns of one head's state; a thread 4 columns and the rows 4 part + 4 PARTS i + e.
// Per token the threads of a column group reduce 4 read-outs (and, delta, 4 recalls S^T k) with a halving exchange: every
// step sends the half of the values the partner keeps, so 8 values over 16 lanes take 8 shuffles instead of 32.
// Tokens are staged 16 at a time; places behind the run's end hold k = q = v = 0, decay 1, strength 0 and change nothing.
constexpr int kScanCols = 32, kScanTokens = 16;

template <int DK, bool DELTA>
struct ScanGeom {
  static constexpr int kParts = DK >= 64 ? 16 : 8;
  static constexpr int kThreads = kParts * (kScanCols / 4);
  static constexpr int kNI = DK / (4 * kParts);
  static constexpr int kK = 0, kQ = kScanTokens * DK, kG = 2 * kScanTokens * DK;       // floats of one staging buffer
  static constexpr int kV = kG + (DELTA ? kScanTokens * DK : 0);
  static constexpr int kTotal = kV + kScanTokens * kScanCols;
};

// Sums NV values over PARTS lanes; lane `part` ends with the total of value (part / (PARTS / NV)).
template <int NV, int PARTS>
__device__ __forceinline__ float halving_sum(float (&v)[NV], int part) {
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
  return v[0];
}

// grid (DV / 32, hv, runs)
template <int DK, int DV, bool DELTA>
__global__ void __launch_bounds__(ScanGeom<DK, DELTA>::kThreads) lin_scan_kernel(LinearArgs a) {
  using G = ScanGeom<DK, DELTA>;
  constexpr int NI = G::kNI, PARTS = G::kParts, NT = G::kThreads;
  constexpr int SHARE_M = PARTS / (DELTA ? 8 : 4);          // lanes that hold one total
  extern __shared__ __align__(16) float sc_smem[];          // [2][G::kTotal]
  __shared__ float qk_s[2][kScanTokens], b_s[2][kScanTokens];
  pdl_wait();
  const int tid = threadIdx.x, cg = tid / PARTS, part = tid % PARTS, lane0 = (tid & 31) - part;
  const int h = blockIdx.y, j0 = blockIdx.x * kScanCols + 4 * cg;
  const int first = a.run_start[blockIdx.z], last = a.run_start[blockIdx.z + 1];
  const int slot = a.row_slot[first];
  const int hk = h / (a.hv / a.hk);
  const PrepView pv = prep_view<DK, DV, DELTA>(a);
  const float dh = DELTA ? 1.f : a.decay[h];
  float* sp = a.state + (static_cast<size_t>(slot) * a.hv + h) * DK * DV + j0;
  const bool fresh = a.positions[first] == 0;
  float s[NI][4][4];                                        // [i][row e][column]
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float4 v = fresh ? make_float4(0.f, 0.f, 0.f, 0.f)
                             : *reinterpret_cast<const float4*>(sp + static_cast<size_t>(4 * PARTS * i + 4 * part + e) * DV);
      s[i][e][0] = v.x; s[i][e][1] = v.y; s[i][e][2] = v.z; s[i][e][3] = v.w;
    }
  auto stage = [&](int buf, int t0) {
    float* b = sc_smem + buf * G::kTotal;
    const int n = min(kScanTokens, last - t0);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), one = make_float4(1.f, 1.f, 1.f, 1.f);
    for (int i = tid; i < kScanTokens * (DK / 4); i += NT) {
      const int tt = i / (DK / 4), c = (i % (DK / 4)) * 4;
      if (tt < n) {
        const size_t o = (static_cast<size_t>(t0 + tt) * a.hk + hk) * DK + c;
        cp_async_16(b + G::kK + tt * DK + c, pv.k + o);
        cp_async_16(b + G::kQ + tt * DK + c, pv.q + o);
        if (DELTA) cp_async_16(b + G::kG + tt * DK + c, pv.g + (static_cast<size_t>(t0 + tt) * a.hv + h) * DK + c);
      } else {
        *reinterpret_cast<float4*>(b + G::kK + tt * DK + c) = zero;
        *reinterpret_cast<float4*>(b + G::kQ + tt * DK + c) = zero;
        if (DELTA) *reinterpret_cast<float4*>(b + G::kG + tt * DK + c) = one;
      }
    }
    for (int i = tid; i < kScanTokens * (kScanCols / 4); i += NT) {
      const int tt = i / (kScanCols / 4), c = (i % (kScanCols / 4)) * 4;
      if (tt < n) cp_async_16(b + G::kV + tt * kScanCols + c, pv.v + (static_cast<size_t>(t0 + tt) * a.hv + h) * DV + blockIdx.x * kScanCols + c);
      else *reinterpret_cast<float4*>(b + G::kV + tt * kScanCols + c) = zero;
    }
    if (tid < kScanTokens) {
      qk_s[buf][tid] = tid < n ? pv.qk[static_cast<size_t>(t0 + tid) * a.hk + hk] : 0.f;
      if (DELTA) b_s[buf][tid] = tid < n ? pv.b[static_cast<size_t>(t0 + tid) * a.hv + h] : 0.f;
    }
    cp_async_group_commit();
  };
  stage(0, first);
  int buf = 0;
  for (int t0 = first; t0 < last; t0 += kScanTokens, buf ^= 1) {
    if (t0 + kScanTokens < last) {
      stage(buf ^ 1, t0 + kScanTokens);
      cp_async_group_wait<1>();
    } else {
      cp_async_group_wait<0>();
    }
    __syncthreads();
    const float* b = sc_smem + buf * G::kTotal;
    const int n = min(kScanTokens, last - t0);
#pragma unroll 4
    for (int tt = 0; tt < kScanTokens; ++tt) {
      float val[DELTA ? 8 : 4];
#pragma unroll
      for (int c = 0; c < (DELTA ? 8 : 4); ++c) val[c] = 0.f;
      float kf[NI][4];
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int r = 4 * PARTS * i + 4 * part;
        const float4 k4 = *reinterpret_cast<const float4*>(b + G::kK + tt * DK + r);
        const float4 q4 = *reinterpret_cast<const float4*>(b + G::kQ + tt * DK + r);
        const float d1 = tt < n ? dh : 1.f;
        float gf[4] = {d1, d1, d1, d1};
        if (DELTA) {
          const float4 g4 = *reinterpret_cast<const float4*>(b + G::kG + tt * DK + r);
          gf[0] = g4.x; gf[1] = g4.y; gf[2] = g4.z; gf[3] = g4.w;
        }
        const float qf[4] = {q4.x, q4.y, q4.z, q4.w};
        kf[i][0] = k4.x; kf[i][1] = k4.y; kf[i][2] = k4.z; kf[i][3] = k4.w;
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            s[i][e][c] *= gf[e];
            if (DELTA) {
              val[c] = fmaf(s[i][e][c], kf[i][e], val[c]);
              val[(DELTA ? 4 : 0) + c] = fmaf(s[i][e][c], qf[e], val[(DELTA ? 4 : 0) + c]);
            } else {
              val[c] = fmaf(s[i][e][c], qf[e], val[c]);
            }
          }
      }
      const float4 v4 = *reinterpret_cast<const float4*>(b + G::kV + tt * kScanCols + 4 * cg);
      float u[4] = {v4.x, v4.y, v4.z, v4.w};
      const float total = halving_sum<DELTA ? 8 : 4, PARTS>(val, part);
      if (DELTA) {
        const float bt = b_s[buf][tt];
#pragma unroll
        for (int c = 0; c < 4; ++c) u[c] = bt * (u[c] - __shfl_sync(0xffffffffu, total, lane0 + c * SHARE_M));
      }
#pragma unroll
      for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < 4; ++c) s[i][e][c] = fmaf(kf[i][e], u[c], s[i][e][c]);
      // the lanes that hold the read-out totals add (q . k) u and store their column
      const int which = part / SHARE_M - (DELTA ? 4 : 0);
      if (which >= 0 && part % SHARE_M == 0 && tt < n) {
        const float uc = which == 0 ? u[0] : (which == 1 ? u[1] : (which == 2 ? u[2] : u[3]));
        a.o[(static_cast<size_t>(t0 + tt) * a.hv + h) * DV + j0 + which] = fmaf(qk_s[buf][tt], uc, total);
      }
    }
    __syncthreads();                                        // this buffer's readers are done before it is staged again
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      *reinterpret_cast<float4*>(sp + static_cast<size_t>(4 * PARTS * i + 4 * part + e) * DV) =
          make_float4(s[i][e][0], s[i][e][1], s[i][e][2], s[i][e][3]);
}

template <typename T, int DK, int DV, bool DELTA>
static int launch_lin(const LinearArgs& a, int decode, cudaStream_t st) {
  using G = LinGeom<DK, DV>;
  if (decode) {
    const size_t smem = static_cast<size_t>(G::kParts) * DV * sizeof(float) * (DELTA ? 2 : 1);
    static_assert(static_cast<size_t>(G::kParts) * DV * 8 <= 48 * 1024, "decode reduction buffer");
    lin_decode_kernel<T, DK, DV, DELTA><<<dim3(a.hv, a.rows), G::kThreads, smem, st>>>(a);
    DGPP_CUDA_OK(cudaGetLastError());
    return 0;
  }
  constexpr size_t smem = 2 * ScanGeom<DK, DELTA>::kTotal * sizeof(float);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(lin_scan_kernel<DK, DV, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    attr = true;
  }
  lin_prep_kernel<T, DK, DV, DELTA><<<dgpp_ceil_div(a.rows * (a.hk + a.hv), 8), 256, 0, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  lin_scan_kernel<DK, DV, DELTA><<<dim3(DV / kScanCols, a.hv, a.runs), ScanGeom<DK, DELTA>::kThreads, smem, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  if (a.conv_w != nullptr) {
    const int C = 2 * a.hk * DK + a.hv * DV;
    lin_tail_kernel<T><<<dim3(dgpp_ceil_div(C, 256), a.runs), 256, 0, st>>>(a, C);
    DGPP_CUDA_OK(cudaGetLastError());
  }
  return 0;
}

template <typename T, bool DELTA>
static int launch_lin_dims(const LinearArgs& a, int DK, int DV, int decode, cudaStream_t st) {
#define DGPP_LIN_CASE(K, V) if (DK == K && DV == V) return launch_lin<T, K, V, DELTA>(a, decode, st);
  DGPP_LIN_CASE(32, 32) DGPP_LIN_CASE(32, 64) DGPP_LIN_CASE(32, 128) DGPP_LIN_CASE(32, 256)
  DGPP_LIN_CASE(64, 32) DGPP_LIN_CASE(64, 64) DGPP_LIN_CASE(64, 128) DGPP_LIN_CASE(64, 256)
  DGPP_LIN_CASE(128, 32) DGPP_LIN_CASE(128, 64) DGPP_LIN_CASE(128, 128) DGPP_LIN_CASE(128, 256)
  DGPP_LIN_CASE(256, 32) DGPP_LIN_CASE(256, 64) DGPP_LIN_CASE(256, 128) DGPP_LIN_CASE(256, 256)
#undef DGPP_LIN_CASE
  dgpp_set_error("linear_state: head widths %d x %d (padded to 32, 64, 128 or 256)", DK, DV);
  return -1;
}

}  // namespace dgpp

using namespace dgpp;

// decode = 1: every row is a run of its own; norm and gate are applied (delta) and `out` is written, or the raw read-outs go
// to `o` (lightning).  decode = 0: the runs named by run_start / row_run0; `o` receives the raw read-outs, prep is scratch
// of rows * (2 hk DK + hv DV + hv DK + hk + hv) floats.  delta = 0: lightning (decay [hv]; hk = hv, no low / A_log / dt_bias).
DGPP_API int dgpp_linear_state(const void* proj, int64_t stride, int c_off, int b_off, const void* low, int64_t low_stride,
                               const void* conv_w, void* ring, int taps, const void* A_log, const void* dt_bias, const void* decay,
                               void* state, const void* row_slot, const void* positions, const void* run_start, const void* row_run0,
                               void* prep, void* o, void* out, int64_t out_stride, const void* norm_w, int rows, int runs, int hk,
                               int hv, int DK, int DV, int vdim, float q_scale, float eps, int delta, int decode, int f32,
                               cudaStream_t st) {
  DGPP_REQUIRE(hk > 0 && hv % hk == 0, "linear_state: %d value heads over %d key heads", hv, hk);
  DGPP_REQUIRE(rows >= 0 && rows <= 65535 && runs <= 65535, "linear_state: %d rows in %d runs", rows, runs);
  DGPP_REQUIRE(conv_w == nullptr || (taps >= 1 && ring), "linear_state: a convolution of %d taps needs its ring", taps);
  DGPP_REQUIRE(!delta || (low && A_log && dt_bias), "linear_state: the delta rule needs its decay inputs");
  DGPP_REQUIRE(delta || (decay && hk == hv), "linear_state: lightning needs a decay per head and as many key heads as heads");
  DGPP_REQUIRE(decode || (run_start && row_run0 && prep && o), "linear_state: runs need their bounds and scratch");
  DGPP_REQUIRE(!decode || (delta ? (out && norm_w) : (o != nullptr)), "linear_state: no output");
  if (rows == 0) return 0;
  LinearArgs a;
  memset(&a, 0, sizeof(a));
  a.proj = proj; a.stride = stride; a.c_off = c_off; a.b_off = b_off;
  a.low = static_cast<const float*>(low); a.low_stride = low_stride;
  a.conv_w = static_cast<const float*>(conv_w); a.ring = static_cast<float*>(ring); a.taps = taps;
  a.A_log = static_cast<const float*>(A_log); a.dt_bias = static_cast<const float*>(dt_bias); a.decay = static_cast<const float*>(decay);
  a.state = static_cast<float*>(state);
  a.row_slot = static_cast<const int32_t*>(row_slot); a.positions = static_cast<const int32_t*>(positions);
  a.run_start = static_cast<const int32_t*>(run_start); a.row_run0 = static_cast<const int32_t*>(row_run0);
  a.prep = static_cast<float*>(prep); a.o = static_cast<float*>(o);
  a.out = out; a.out_stride = out_stride; a.norm_w = static_cast<const float*>(norm_w);
  a.rows = rows; a.runs = runs; a.hk = hk; a.hv = hv; a.vdim = vdim; a.q_scale = q_scale; a.eps = eps;
  if (f32) return delta ? launch_lin_dims<float, true>(a, DK, DV, decode, st) : launch_lin_dims<float, false>(a, DK, DV, decode, st);
  return delta ? launch_lin_dims<bf16, true>(a, DK, DV, decode, st) : launch_lin_dims<bf16, false>(a, DK, DV, decode, st);
}

// GQA for prompt rows on the 5th-generation tensor cores (bf16 queries, keys and values; see window_attn.cuh for the layer, its windows,
// chunks and maps, and for the cache, whose new positions and prepared queries `qk_norm_append` has written).
//
// One CTA = 128 query rows of one key head: 128 / G consecutive tokens of one run with their G = hq / hkv query heads, row
// r = token r / G, head r % G (differential attention: `maps` key heads read the same values; finished fp32 outputs go to `raw`).  It walks the cache pages from the first key its first token sees to its last token:
//
//   MMA1     S[r, t] = q_r . k_t              (fp32 in TMEM, double buffered: tile i + 1 overlaps the softmax of tile i)
//   softmax  one thread per row: running maximum, p = 2^(s - m), window and causal mask; p goes to shared memory as two
//            bf16 terms (value + residual), so the weights keep 16 bits of mantissa through the tensor core
//   MMA2     O[r, :] += p_hi V + p_lo V       (fp32 in TMEM over all tiles)
//
// O stays in TMEM: it is rescaled only when a row's maximum grew by more than 8 binary orders since the last time.  Until
// then the exponents are taken against the older maximum, for the weights and for their sum alike, so the quotient is the
// softmax either way.
// Warps: 0 = TMA producer (one page of keys and values per stage), 1 = MMA issuer / TMEM owner, 2..5 = softmax.
//
// EXT: kept first tokens, whose pages come before those of the window; a sink, which joins the sum of the weights at the end; rotated values,
// turned back there too, columns m and m + DV / 2 of a row together.  CAP: scores pass cap * tanh(s / cap) as well; caps of up to 38
// bound the exponents by 110 binary orders, so the cap itself stands for the maximum and nothing is ever rescaled.
//
// FLAT is the form for latent attention, whose keys and values are expanded from the cached latents before the launch: every head
// is its own kv head; key columns 0 .. DN - 1 and the values come from the expanded rows [flat rows, hq * DN + hq * DV], the other
// key columns (the rotated part that all heads share) from the gathered cache rows.  A run's page g starts at flat row
// flat_base[run] + 64 g.  An output gate per (row, head) may multiply the result.
// Every wait is bounded; on expiry the kernel records a status code and unwinds.
#include <cuda.h>
#include <math.h>
#include <string.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"
#include "kernels/gemm_common.cuh"

namespace dgpp {

constexpr int kWtThreads = 192, kWtRows = 128, kWtKeys = 64;

struct WindowTcParams {
  const bf16* proj;         // [rows, stride], normed query head h at column q_off + h * D
  int64_t stride;
  int q_off;
  const int32_t* block_table;
  const int32_t* row_req;
  const int32_t* positions;
  const int32_t* run_start; // [runs + 1], or [runs] with run_len
  const int32_t* run_len;   // optional [runs]: the runs are not back to back
  const int32_t* flat_base; // [runs] (FLAT)
  const bf16* gate;         // optional [rows, stride]: sigmoid(gate[row, head]) multiplies the output
  float* raw;               // optional [rows, hq, DV] fp32: the outputs instead of `out`
  bf16* out;
  int64_t out_stride;
  DeviceStatus* status;
  int runs, hq, hkv, maps, D, DV, max_blocks, window, chunked, stages;   // hkv: key heads; value heads: hkv / maps
  const float* sink;        // optional [hq]: exp(sink) joins the sum of a row's weights
  const float2* turn;       // optional [rows, DV / 2]: cosines and sines by which a row's outputs are turned back
  int keep_first;           // positions below are seen from everywhere
  float softcap;            // CAP
  int DN, rot_col;          // FLAT: key columns from the expanded rows; first rotated column of a gathered cache row
  float scale, out_scale;
};

__device__ __forceinline__ uint32_t wt_sw128(uint32_t row, uint32_t byte_in_row) {
  return row * 128u + ((((byte_in_row >> 4) ^ (row & 7u)) << 4) | (byte_in_row & 15u));
}

// First position that the query at position i sees
__device__ __forceinline__ int wt_first_key(const WindowTcParams& p, int i) { return p.chunked ? i - i % p.window : max(0, i + 1 - p.window); }

// Largest masked score of 64 keys (row of this thread); keys below `keep` are seen although they lie before lo
template <bool kMask, bool EXT>
__device__ __forceinline__ float wt_row_max(uint32_t taddr, int t0, int lo, int hi, int keep) {
  float mt = -INFINITY;
#pragma unroll
  for (int c0 = 0; c0 < kWtKeys; c0 += 16) {
    uint32_t raw[16];
    tmem_ld_x16(taddr + c0, raw);
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int t = t0 + c0 + j;
      mt = fmaxf(mt, (!kMask || (t <= hi && (t >= lo || (EXT && t < keep)))) ? __uint_as_float(raw[j]) : -INFINITY);
    }
  }
  return mt;
}

// cap * tanh(s / cap) in binary orders: top - 2 top / (1 + 2^(s in)), in = 2 scale log2(e) / cap, top = cap log2(e)
__device__ __forceinline__ float wt_cap(float s, float in, float top) { return top - __fdividef(2.f * top, 1.f + fast_exp2(s * in)); }

// p = 2^(s * sm - m) (CAP: 2^(wt_cap(s, sm, top) - m)) as two bf16 terms into row r of the A operand; returns the row's sum
template <bool kMask, bool EXT, bool CAP>
__device__ __forceinline__ float wt_probs(uint32_t taddr, unsigned char* sP, int r, float sm, float top, float neg_m, int t0, int lo, int hi, int keep) {
  float sum = 0.f;
#pragma unroll
  for (int c0 = 0; c0 < kWtKeys; c0 += 16) {
    uint32_t raw[16];
    tmem_ld_x16(taddr + c0, raw);
    Pack16 a[2], b[2];
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int t = t0 + c0 + j;
      const float s = __uint_as_float(raw[j]);
      const float p = (!kMask || (t <= hi && (t >= lo || (EXT && t < keep)))) ? fast_exp2(CAP ? wt_cap(s, sm, top) + neg_m : fmaf(s, sm, neg_m)) : 0.f;
      sum += p;
      const bf16 h = f32_to_bf16(p);
      a[j >> 3].h[j & 7] = h;
      b[j >> 3].h[j & 7] = f32_to_bf16(p - bf16_to_f32(h));
    }
#pragma unroll
    for (int v = 0; v < 2; ++v) {
      *reinterpret_cast<uint4*>(sP + wt_sw128(r, c0 * 2 + v * 16)) = a[v].u;
      *reinterpret_cast<uint4*>(sP + kWtRows * 128 + wt_sw128(r, c0 * 2 + v * 16)) = b[v].u;
    }
  }
  return sum;
}

// grid (tiles of all runs, hkv)
template <bool FLAT, bool EXT, bool CAP>
__global__ void __launch_bounds__(kWtThreads, 1)
window_attn_tc_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, WindowTcParams p) {
  extern __shared__ __align__(1024) unsigned char smem_dyn[];
  const int kblk = kWtKeys * 128;                              // 64 keys x 64 columns, one swizzle atom column
  const int natom = p.D / 64, vatom = p.DV / 64;
  unsigned char* sp = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_dyn) + 1023) & ~uintptr_t(1023));
  unsigned char* sQ = sp;  sp += natom * kWtRows * 128;
  unsigned char* sP = sp;  sp += 2 * kWtRows * 128;            // value term, residual term
  unsigned char* sK = sp;  sp += p.stages * natom * kblk;
  unsigned char* sV = sp;  sp += p.stages * vatom * kblk;
  uint64_t* kv_full = reinterpret_cast<uint64_t*>(sp);         // [4]
  uint64_t* kv_empty = kv_full + 4;                            // [4]
  uint64_t* s_full = kv_empty + 4;                             // [2]
  uint64_t* p_full = s_full + 2;
  uint64_t* o_full = p_full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int group = p.hq / p.hkv, per = kWtRows / group, kvh = blockIdx.y;
  const uint32_t tmem_cols = p.DV <= 128 ? 256u : 512u;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 4; ++i) { mbar_init(&kv_full[i], 1); mbar_init(&kv_empty[i], 1); }
    mbar_init(&s_full[0], 1); mbar_init(&s_full[1], 1);
    mbar_init(p_full, 4);
    mbar_init(o_full, 1);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  pdl_wait();
  // the run this tile lies in (tiles are dealt run by run)
  int tile = blockIdx.x, row0 = 0, ntok = 0, flat0 = 0;
  for (int r = 0; r < p.runs; ++r) {
    const int a = p.run_start[r], n = p.run_len != nullptr ? p.run_len[r] : p.run_start[r + 1] - a, t = (n + per - 1) / per;
    if (tile < t) {
      row0 = a + tile * per;
      ntok = min(per, n - tile * per);
      if (FLAT) flat0 = p.flat_base[r];
      break;
    }
    tile -= t;
  }
  const int first_pos = p.positions[row0], last_pos = first_pos + ntok - 1;
  const int32_t* bt = p.block_table + static_cast<size_t>(p.row_req[row0]) * p.max_blocks;
  // pages in order: those of the kept first tokens, then from the first one that the window of the tile's first token reaches
  const int page0 = wt_first_key(p, first_pos) / kWtKeys, nkeep = EXT ? min((p.keep_first + kWtKeys - 1) / kWtKeys, page0) : 0;
  const int ntiles = ntok > 0 ? last_pos / kWtKeys - page0 + 1 + nkeep : 0;
  auto page_of = [&](int i) { return EXT && i < nkeep ? i : page0 - nkeep + i; };
  if (warp >= 2) {
    // ---- this thread's query row into the swizzled A operand
    const int r = (warp & 3) * 32 + lane, tok = r / group;
    const bool live = tok < ntok;
    const uint4* src = reinterpret_cast<const uint4*>(p.proj + static_cast<size_t>(row0 + (live ? tok : 0)) * p.stride + p.q_off +
                                                      (kvh * group + r % group) * p.D);
    for (int c = 0; c < p.D / 8; ++c) {
      const uint4 v = live ? src[c] : make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(sQ + (c >> 3) * kWtRows * 128 + wt_sw128(r, (c & 7) * 16)) = v;
    }
    fence_proxy_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 2 * kWtKeys;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (elect_one()) {
      for (int i = 0; i < ntiles; ++i) {
        const int s = i % p.stages;
        if (!wait_bar(&kv_empty[s], ((i / p.stages) & 1) ^ 1)) { report(p.status, kTimeoutStageEmpty, 71); *abort_flag = 1; break; }
        mbar_expect_tx(&kv_full[s], (natom + vatom) * kblk);
        if (FLAT) {                              // tmK: expanded rows, tmV: gathered cache rows
          const int y = flat0 + page_of(i) * kWtKeys, nn = p.DN / 64;
          for (int a = 0; a < nn; ++a) tma_load_2d(sK + (s * natom + a) * kblk, &tmK, kvh * p.DN + a * 64, y, &kv_full[s]);
          for (int a = nn; a < natom; ++a) tma_load_2d(sK + (s * natom + a) * kblk, &tmV, p.rot_col + (a - nn) * 64, y, &kv_full[s]);
          for (int a = 0; a < vatom; ++a) tma_load_2d(sV + (s * vatom + a) * kblk, &tmK, p.hq * p.DN + kvh * p.DV + a * 64, y, &kv_full[s]);
        } else {
          const int pg = bt[page_of(i)], y = (pg * p.hkv + kvh) * kWtKeys, yv = (pg * (p.hkv / p.maps) + kvh / p.maps) * kWtKeys;
          for (int a = 0; a < natom; ++a) tma_load_2d(sK + (s * natom + a) * kblk, &tmK, a * 64, y, &kv_full[s]);
          for (int a = 0; a < vatom; ++a) tma_load_2d(sV + (s * vatom + a) * kblk, &tmV, a * 64, yv, &kv_full[s]);
        }
        if (*abort_flag) break;
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      const uint32_t idesc1 = umma_idesc_f16(kWtRows, kWtKeys, 1u, 1u);                // Q (K-major) x K (K-major)
      const uint32_t idesc2 = umma_idesc_f16(kWtRows, p.DV, 1u, 1u) | (1u << 16);      // P (K-major) x V (MN-major B)
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      auto mma2 = [&](int j) {
        const int s = j % p.stages;
        const uint32_t v_addr = smem_u32(sV + s * vatom * kblk);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int k = 0; k < kWtKeys / 16; ++k)   // 16 keys per step: P advances 32 bytes, V two 8-row groups
            umma_f16(tmem_o, umma_desc_sw128(p_addr + term * kWtRows * 128 + k * 32), umma_desc_sw128_mn(v_addr + k * 2048, kblk),
                     idesc2, (j > 0 || term > 0 || k > 0) ? 1u : 0u);
        umma_commit(o_full);
        umma_commit(&kv_empty[s]);
      };
      bool ok = true;
      for (int i = 0; i < ntiles && ok; ++i) {
        const int s = i % p.stages, b = i & 1;
        if (!wait_bar(&kv_full[s], (i / p.stages) & 1)) { report(p.status, kTimeoutTmaFull, 72); *abort_flag = 1; ok = false; break; }
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + s * natom * kblk);
        for (int a = 0; a < natom; ++a)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16(tmem_s + b * kWtKeys, umma_desc_sw128(q_addr + a * kWtRows * 128 + k * 32), umma_desc_sw128(k_addr + a * kblk + k * 32),
                     idesc1, (a > 0 || k > 0) ? 1u : 0u);
        umma_commit(&s_full[b]);
        if (i > 0) {
          if (!wait_bar(p_full, (i - 1) & 1)) { report(p.status, kTimeoutConvert, 73); *abort_flag = 1; ok = false; break; }
          tc_fence_after();
          mma2(i - 1);
        }
        if (*abort_flag) ok = false;
      }
      if (ok && ntiles > 0) {
        if (wait_bar(p_full, (ntiles - 1) & 1)) {
          tc_fence_after();
          mma2(ntiles - 1);
        } else {
          report(p.status, kTimeoutConvert, 74);
          *abort_flag = 1;
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax (thread = query row)
    const int quad = warp & 3, r = quad * 32 + lane, tok = r / group;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const bool live = tok < ntok;
    const int hi = first_pos + (live ? tok : 0), lo = wt_first_key(p, hi);
    const float log2e = 1.4426950408889634f, top = CAP ? p.softcap * log2e : 0.f;
    const float sm = CAP ? 2.f * p.scale * log2e / p.softcap : p.scale * log2e;
    const int keep = EXT ? p.keep_first : 0;
    const bool bounded = CAP && top <= 55.f;
    float m_used = bounded ? top : -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int i = 0; i < ntiles; ++i) {
      const int b = i & 1, t0 = page_of(i) * kWtKeys;
      ok = __all_sync(0xffffffffu, wait_bar(&s_full[b], (i >> 1) & 1) && !*abort_flag) != 0;
      if (!ok) { report(p.status, kTimeoutAccum, 75); *abort_flag = 1; break; }
      tc_fence_after();
      // warp-uniform choices: the TMEM accesses are .sync.aligned
      const bool full = __all_sync(0xffffffffu, t0 + kWtKeys - 1 <= hi && (t0 >= lo || (EXT && t0 + kWtKeys <= keep))) != 0;
      const float mt = bounded ? -INFINITY : full ? wt_row_max<false, EXT>(tmem_s + b * kWtKeys + lane_addr, t0, lo, hi, keep)
                            : wt_row_max<true, EXT>(tmem_s + b * kWtKeys + lane_addr, t0, lo, hi, keep);
      const float mn = fmaxf(m_used, mt == -INFINITY ? -INFINITY : (CAP ? wt_cap(mt, sm, top) : mt * sm));
      const bool grow = mn > m_used + 8.f || (m_used == -INFINITY && mn != -INFINITY);
      if (i > 0) {
        // the previous tile's product is complete: its weights may be overwritten, O may be rescaled
        ok = __all_sync(0xffffffffu, wait_bar(o_full, (i - 1) & 1)) != 0;
        if (!ok) { report(p.status, kTimeoutAccum, 76); *abort_flag = 1; break; }
        tc_fence_after();
      }
      if (__any_sync(0xffffffffu, grow)) {
        const float corr = !grow ? 1.f : (m_used == -INFINITY ? 0.f : fast_exp2(m_used - mn));
        if (grow) m_used = mn;
        l_run *= corr;
        if (i > 0) {
          for (int c0 = 0; c0 < p.DV; c0 += 16) {
            uint32_t raw[16];
            tmem_ld_x16(tmem_o + lane_addr + c0, raw);
#pragma unroll
            for (int j = 0; j < 16; ++j) raw[j] = __float_as_uint(__uint_as_float(raw[j]) * corr);
            tmem_st_x16(tmem_o + lane_addr + c0, raw);
          }
        }
      }
      const float neg_m = m_used == -INFINITY ? 0.f : -m_used;
      l_run += full ? wt_probs<false, EXT, CAP>(tmem_s + b * kWtKeys + lane_addr, sP, r, sm, top, neg_m, t0, lo, hi, keep)
                    : wt_probs<true, EXT, CAP>(tmem_s + b * kWtKeys + lane_addr, sP, r, sm, top, neg_m, t0, lo, hi, keep);
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    if (ok && ntiles > 0) {
      ok = __all_sync(0xffffffffu, wait_bar(o_full, (ntiles - 1) & 1) && !*abort_flag) != 0;
      if (!ok) {
        report(p.status, kTimeoutAccum, 77);
        *abort_flag = 1;
      } else {
        tc_fence_after();
        if (EXT && p.sink != nullptr && l_run > 0.f) l_run += fast_exp2(fmaf(p.sink[kvh * group + r % group], log2e, -m_used));
        float f = l_run > 0.f ? p.out_scale / l_run : 0.f;
        if (p.gate != nullptr && live) f *= sigmoid_f32(bf16_to_f32(p.gate[static_cast<size_t>(row0 + tok) * p.stride + kvh * group + r % group]));
        float* dst32 = p.raw != nullptr ? p.raw + (static_cast<size_t>(row0 + (live ? tok : 0)) * p.hq + kvh * group + r % group) * p.DV : nullptr;
        bf16* dst = p.out + static_cast<size_t>(row0 + (live ? tok : 0)) * p.out_stride + static_cast<size_t>(kvh * group + r % group) * p.DV;
        const int half = p.DV / 2;
        const float2* turn = EXT && p.turn != nullptr ? p.turn + static_cast<size_t>(row0 + (live ? tok : 0)) * half : nullptr;
        for (int c0 = 0; c0 < p.DV; c0 += 16) {
          uint32_t raw[16];
          if (EXT && turn != nullptr) {                                 // 16 columns of both halves (DV / 2 is a multiple of 32)
            if (c0 >= half) break;
            uint32_t other[16];
            tmem_ld_x16(tmem_o + lane_addr + c0, raw);
            tmem_ld_x16(tmem_o + lane_addr + half + c0, other);
            if (live) {
              Pack16 o[2], q[2];
#pragma unroll
              for (int j = 0; j < 16; ++j) {
                const float2 cs = turn[c0 + j];
                const float a = __uint_as_float(raw[j]) * f, b = __uint_as_float(other[j]) * f;
                o[j >> 3].h[j & 7] = f32_to_bf16(fmaf(b, cs.y, a * cs.x));
                q[j >> 3].h[j & 7] = f32_to_bf16(fmaf(-a, cs.y, b * cs.x));
              }
              *reinterpret_cast<uint4*>(dst + c0) = o[0].u;
              *reinterpret_cast<uint4*>(dst + c0 + 8) = o[1].u;
              *reinterpret_cast<uint4*>(dst + half + c0) = q[0].u;
              *reinterpret_cast<uint4*>(dst + half + c0 + 8) = q[1].u;
            }
            continue;
          }
          tmem_ld_x16(tmem_o + lane_addr + c0, raw);
          if (live && dst32 != nullptr) {
#pragma unroll
            for (int j = 0; j < 16; j += 4)
              *reinterpret_cast<float4*>(dst32 + c0 + j) = make_float4(__uint_as_float(raw[j]) * f, __uint_as_float(raw[j + 1]) * f,
                                                                     __uint_as_float(raw[j + 2]) * f, __uint_as_float(raw[j + 3]) * f);
          } else if (live) {
            Pack16 o[2];
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j >> 3].h[j & 7] = f32_to_bf16(__uint_as_float(raw[j]) * f);
            *reinterpret_cast<uint4*>(dst + c0) = o[0].u;
            *reinterpret_cast<uint4*>(dst + c0 + 8) = o[1].u;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, tmem_cols);
}

}  // namespace dgpp

using namespace dgpp;

static int wt_check(const void* proj, int64_t stride, int q_off, const void* out, int64_t out_stride, int runs, int hq, int hkv, int D, int DV,
                    int page, int window) {                    // hkv: key heads
  DGPP_REQUIRE(hkv > 0 && hq % hkv == 0 && hq / hkv <= kWtRows, "window_attn_tc: %d query heads over %d key heads", hq, hkv);
  DGPP_REQUIRE(D % 64 == 0 && D >= 64 && D <= 256 && DV % 64 == 0 && DV >= 64 && DV <= 256, "window_attn_tc: head widths %d / %d", D, DV);
  DGPP_REQUIRE(page == kWtKeys, "window_attn_tc: page %d (64)", page);
  DGPP_REQUIRE(stride % 8 == 0 && q_off % 8 == 0 && out_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(out) & 15) == 0, "window_attn_tc: rows must be 16-byte aligned");
  DGPP_REQUIRE(window >= 1 && runs >= 1, "window_attn_tc: window %d, %d runs", window, runs);
  return 0;
}

template <bool FLAT, bool EXT, bool CAP>
static int launch_wt(const CUtensorMap& tK, const CUtensorMap& tV, WindowTcParams& p, int tiles, cudaStream_t st) {
  const size_t fixed = 1024 + static_cast<size_t>(p.D / 64 + 2) * kWtRows * 128 + 192, stage = static_cast<size_t>(p.D + p.DV) * 128;
  const size_t limit = 227 * 1024;
  p.stages = static_cast<int>((limit - fixed) / stage);
  p.stages = p.stages > 4 ? 4 : p.stages;
  DGPP_REQUIRE(p.stages >= 2, "window_attn_tc: head widths %d / %d do not fit shared memory", p.D, p.DV);
  static bool attr = false;
  if (!attr) {
    DGPP_CUDA_OK(cudaFuncSetAttribute(window_attn_tc_kernel<FLAT, EXT, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(limit)));
    attr = true;
  }
  window_attn_tc_kernel<FLAT, EXT, CAP><<<dim3(tiles, p.hkv), kWtThreads, fixed + p.stages * stage, st>>>(tK, tV, p);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// Runs of consecutive rows (run_start [runs + 1], or run_start / run_len [runs]); `tiles` = sum over the runs of ceil(length / (128 /
// group)), group = hq / (hkv * maps).  The cache (pages of 64 tokens) holds the runs' own positions already.  chunked: `window` is the
// size of the chunks.  gate_off >= 0: the sigmoid of that column of a row, one per head, multiplies the head's output.  raw: fp32
// outputs [rows, hq, DV] instead of `out`.  sink [hq], turn [rows, DV / 2] pairs (see qk_norm_append): optional; keep_first: that many first
// positions are seen from everywhere; softcap 0: none.
DGPP_API int dgpp_window_attn_tc(const void* proj, int64_t stride, int q_off, const void* k_cache, const void* v_cache,
                                 const void* block_table, const void* row_req, const void* positions, const void* run_start, const void* run_len,
                                 void* out, int64_t out_stride, void* raw, int runs, int tiles, int hq, int hkv, int maps, int D, int DV, int page,
                                 int max_blocks, int num_blocks, int window, int chunked, int gate_off, float scale, float out_scale,
                                 const void* sink, const void* turn, int keep_first, float softcap, cudaStream_t st) {
  DGPP_REQUIRE(maps == 1 || (maps == 2 && raw && !sink), "window_attn_tc: %d maps", maps);
  DGPP_REQUIRE(!turn || !raw, "window_attn_tc: fp32 outputs are not turned back");
  DGPP_REQUIRE(keep_first >= 0 && (!chunked || keep_first == 0) && softcap >= 0.f, "window_attn_tc: %d kept tokens, cap %f", keep_first, static_cast<double>(softcap));
  if (wt_check(proj, stride, q_off, out, out_stride, runs, hq, hkv * maps, D, DV, page, window)) return -1;
  if (tiles == 0) return 0;
  WindowTcParams p;
  memset(&p, 0, sizeof(p));
  p.proj = static_cast<const bf16*>(proj); p.stride = stride; p.q_off = q_off;
  p.block_table = static_cast<const int32_t*>(block_table);
  p.row_req = static_cast<const int32_t*>(row_req);
  p.positions = static_cast<const int32_t*>(positions);
  p.run_start = static_cast<const int32_t*>(run_start);
  p.run_len = static_cast<const int32_t*>(run_len);
  p.gate = gate_off >= 0 ? p.proj + gate_off : nullptr;
  p.raw = static_cast<float*>(raw);
  p.out = static_cast<bf16*>(out); p.out_stride = out_stride;
  p.status = device_status_ptr();
  p.runs = runs; p.hq = hq; p.hkv = hkv * maps; p.maps = maps; p.chunked = chunked; p.D = D; p.DV = DV; p.max_blocks = max_blocks; p.window = window;
  p.scale = scale; p.out_scale = out_scale;
  p.sink = static_cast<const float*>(sink); p.turn = static_cast<const float2*>(turn); p.keep_first = keep_first; p.softcap = softcap;
  const uint64_t rows = static_cast<uint64_t>(num_blocks) * hkv * page;
  CUtensorMap tK, tV;
  if (make_tmap_2d(&tK, k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, D, rows * maps, static_cast<uint64_t>(D) * 2, 64, kWtKeys, CU_TENSOR_MAP_SWIZZLE_128B))
    return -1;
  if (make_tmap_2d(&tV, v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, DV, rows, static_cast<uint64_t>(DV) * 2, 64, kWtKeys, CU_TENSOR_MAP_SWIZZLE_128B))
    return -1;
  if (p.softcap > 0.f) return launch_wt<false, true, true>(tK, tV, p, tiles, st);
  const bool ext = p.sink != nullptr || p.turn != nullptr || p.keep_first > 0;
  return ext ? launch_wt<false, true, false>(tK, tV, p, tiles, st) : launch_wt<false, false, false>(tK, tV, p, tiles, st);
}

// The same over keys and values expanded from a latent cache: `flat` [flat_rows, heads * (dn + dv)] bf16, `lat` [flat_rows, lat_cols]
// bf16 (the gathered cache rows, rotated key part from column rot_col), query head h at q_off + h * (dn + dr) of its row.  Runs:
// run_start / run_len [runs]; flat row of position 0 of a run: flat_base (may be negative).  gate_off >= 0: sigmoid of that column
// of a row, one per head, multiplies the head's output.
DGPP_API int dgpp_latent_prefill_tc(const void* proj, int64_t stride, int q_off, int gate_off, const void* flat, const void* lat, int lat_cols,
                                    int rot_col, const void* row_req, const void* positions, const void* run_start, const void* run_len,
                                    const void* flat_base, void* out, int64_t out_stride, int runs, int tiles, int flat_rows, int heads, int dn,
                                    int dr, int dv, int window, float scale, cudaStream_t st) {
  if (wt_check(proj, stride, q_off, out, out_stride, runs, heads, heads, dn + dr, dv, kWtKeys, window)) return -1;
  DGPP_REQUIRE(dn % 64 == 0 && dn >= 64 && dr % 64 == 0 && dr >= 0 && lat_cols % 8 == 0 && rot_col % 8 == 0 && rot_col + dr <= lat_cols,
               "latent_prefill_tc: key widths %d + %d, cache rows of %d", dn, dr, lat_cols);
  DGPP_REQUIRE(run_len && flat_base && flat_rows % kWtKeys == 0, "latent_prefill_tc: %d flat rows", flat_rows);
  if (tiles == 0) return 0;
  WindowTcParams p;
  memset(&p, 0, sizeof(p));
  p.proj = static_cast<const bf16*>(proj); p.stride = stride; p.q_off = q_off;
  p.row_req = static_cast<const int32_t*>(row_req);
  p.positions = static_cast<const int32_t*>(positions);
  p.run_start = static_cast<const int32_t*>(run_start);
  p.run_len = static_cast<const int32_t*>(run_len);
  p.flat_base = static_cast<const int32_t*>(flat_base);
  p.gate = gate_off >= 0 ? p.proj + gate_off : nullptr;
  p.out = static_cast<bf16*>(out); p.out_stride = out_stride;
  p.status = device_status_ptr();
  p.runs = runs; p.hq = heads; p.hkv = heads; p.maps = 1; p.D = dn + dr; p.DV = dv; p.window = window;
  p.DN = dn; p.rot_col = rot_col;
  p.scale = scale; p.out_scale = 1.f;
  const uint64_t cols = static_cast<uint64_t>(heads) * (dn + dv);
  CUtensorMap tK, tV;
  if (make_tmap_2d(&tK, flat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, cols, flat_rows, cols * 2, 64, kWtKeys, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
  if (make_tmap_2d(&tV, lat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, lat_cols, flat_rows, static_cast<uint64_t>(lat_cols) * 2, 64, kWtKeys, CU_TENSOR_MAP_SWIZZLE_128B)) return -1;
  return launch_wt<true, false, false>(tK, tV, p, tiles, st);
}

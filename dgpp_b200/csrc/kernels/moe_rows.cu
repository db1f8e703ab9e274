// Mixture of experts over plain 16-bit or 32-bit rows (expert matrices without block scales): the launches between the router
// logits and the grouped linears.
//
//   moe_route_small    up to 16 tokens, one CTA: picks every token's experts from its logits (sigmoid or softmax weights, ties to
//                      the lower id), lists the experts in use as tiles of 16 rows over the SAME activation rows, and writes the
//                      row of every (token, choice) pair and every tile row's weight (0: the token did not choose the expert);
//                      choices at or beyond `experts` are identity experts, whose output is the token's input: row -1
//   moe_scatter_rows   any number of tokens, after the counting sort of moe_prefill.cu: copies a pair's activation row to its place
//                      in the sorted tiles and writes the row's weight there
// The weights ride along per tile row, so the activation kernel can scale what an expert sees.
#include <math.h>

#include "common/common.h"
#include "common/dtypes.cuh"
#include "common/elem.cuh"
#include "common/ptx.cuh"

namespace dgpp {

constexpr int kSmallTokens = 16, kSmallExperts = 512, kSmallTop = 16, kSmallThreads = kSmallTokens * 32;

struct RouteSmall {
  const float* logits;     // [T, stride]
  int64_t stride;
  int32_t* pair_row;       // [T * top]
  int32_t* tiles;          // [max_tiles]
  float* row_w;            // [max_tiles * 16]
  float* wts;              // [T * top] weight of every pair, or null
  const float* bias;       // [E] added to the logits, or null
  const float* correction; // [E] added to the scores for the choice alone, or null
  int T, E, top, max_tiles, score;   // score: 0 sigmoid, 1 softmax over all experts, 2 softmax over the chosen ones
  int experts, norm_topk;            // outputs with matrices (the others are identity experts); weights divided by their sum
};

__global__ void __launch_bounds__(kSmallThreads) moe_route_small_kernel(RouteSmall a) {
  __shared__ int slot[kSmallExperts];
  __shared__ int ids[kSmallTokens][kSmallTop];
  __shared__ float wts[kSmallTokens][kSmallTop];
  __shared__ int warp_cnt[kSmallTokens];
  pdl_wait();
  const int tid = threadIdx.x, t = tid >> 5, lane = tid & 31;
  for (int e = tid; e < kSmallExperts; e += kSmallThreads) slot[e] = 0;
  for (int i = tid; i < a.max_tiles * kSmallTokens; i += kSmallThreads) a.row_w[i] = 0.f;
  __syncthreads();
  if (t < a.T) {
    float z[kSmallExperts / 32];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < kSmallExperts / 32; ++i) {
      const int e = lane + 32 * i;
      z[i] = e < a.E ? a.logits[t * a.stride + e] + (a.bias != nullptr ? a.bias[e] : 0.f) : -INFINITY;
      mx = fmaxf(mx, z[i]);
    }
    float norm = 1.f;
    if (a.score == 1) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kSmallExperts / 32; ++i) sum += expf(z[i] - mx);
      norm = warp_sum_f32(sum);
    }
    // with a correction the choice goes by score + correction, and the scores are kept
    float sc[kSmallExperts / 32];
    if (a.correction != nullptr) {
#pragma unroll
      for (int i = 0; i < kSmallExperts / 32; ++i) {
        const int e = lane + 32 * i;
        if (e >= a.E) continue;
        sc[i] = a.score == 0 ? sigmoid_f32(z[i]) : expf(z[i] - mx) / norm;
        z[i] = sc[i] + a.correction[e];
      }
    }
    // both scores grow with the logit; equal scores of different logits go to the larger logit
    for (int r = 0; r < a.top; ++r) {
      float bv = -INFINITY;
      int be = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < kSmallExperts / 32; ++i) {
        const int e = lane + 32 * i;
        if (e < a.E && (z[i] > bv || (z[i] == bv && e < be))) { bv = z[i]; be = e; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
      }
      if (be >= a.E) be = 0;                           // only with logits that are not numbers
      float chosen = 0.f;
#pragma unroll
      for (int i = 0; i < kSmallExperts / 32; ++i)
        if (lane + 32 * i == be) {
          z[i] = -INFINITY;
          if (a.correction != nullptr) chosen = sc[i];
        }
      if (a.correction != nullptr) chosen = __shfl_sync(0xffffffffu, chosen, be & 31);
      if (lane == 0) {
        int j = r;                                     // ascending ids: the order of the sum
        while (j > 0 && ids[t][j - 1] > be) { ids[t][j] = ids[t][j - 1]; wts[t][j] = wts[t][j - 1]; --j; }
        ids[t][j] = be;
        if (r == 0 && a.score == 2) mx = bv;           // the largest comes first
        wts[t][j] = a.correction != nullptr ? chosen : (a.score == 0 ? sigmoid_f32(bv) : expf(bv - mx) / norm);
        if (be < a.experts) slot[be] = 1;
      }
    }
    if ((a.score == 2 || a.norm_topk) && lane == 0) {
      float sum = 1e-20f;
      for (int j = 0; j < a.top; ++j) sum += wts[t][j];
      for (int j = 0; j < a.top; ++j) wts[t][j] /= sum;
    }
  }
  __syncthreads();
  // experts in use, ascending (one thread per expert)
  const bool on = slot[tid] != 0;
  const unsigned bal = __ballot_sync(0xffffffffu, on);
  if (lane == 0) warp_cnt[t] = __popc(bal);
  __syncthreads();
  int at = __popc(bal & ((1u << lane) - 1u)), total = 0;
  for (int w = 0; w < kSmallTokens; ++w) {
    if (w < t) at += warp_cnt[w];
    total += warp_cnt[w];
  }
  slot[tid] = at;
  if (on && at < a.max_tiles) a.tiles[at] = tid;
  for (int i = total + tid; i < a.max_tiles; i += kSmallThreads) a.tiles[i] = -1;
  __syncthreads();
  if (t < a.T && lane < a.top) {
    if (a.wts != nullptr) a.wts[t * a.top + lane] = wts[t][lane];
    if (ids[t][lane] >= a.experts) {
      a.pair_row[t * a.top + lane] = -1;
    } else {
      const int row = min(slot[ids[t][lane]], a.max_tiles - 1) * kSmallTokens + t;
      a.pair_row[t * a.top + lane] = row;
      a.row_w[row] = wts[t][lane];
    }
  }
}

// grid (T * top), 128 threads
template <typename T>
__global__ void __launch_bounds__(128) moe_scatter_rows_kernel(const T* __restrict__ x, const int32_t* __restrict__ pair_row,
                                                               const float* __restrict__ weights, T* __restrict__ xs, float* __restrict__ row_w,
                                                               int cols, int top) {
  pdl_wait();
  const size_t p = blockIdx.x;
  const int row = pair_row[p];
  if (row < 0) return;
  const uint4* src = reinterpret_cast<const uint4*>(x + (p / top) * cols);
  uint4* dst = reinterpret_cast<uint4*>(xs + static_cast<size_t>(row) * cols);
  const int n = cols * static_cast<int>(sizeof(T)) / 16;
  for (int i = threadIdx.x; i < n; i += 128) dst[i] = src[i];
  if (threadIdx.x == 0) row_w[row] = weights[p];
}

}  // namespace dgpp

using namespace dgpp;

// logits [T, E] fp32 with row stride `stride` (bias [E] fp32 or null is added), T <= 16.  The first `experts` outputs have matrices;
// max_tiles >= min(experts, T * top).  correction [E] or null: added to the scores for the choice alone; norm_topk: weights divided by
// their sum.  wts [T * top] or null: the pairs' weights.
DGPP_API int dgpp_moe_route_small(const void* logits, int64_t stride, const void* bias, const void* correction, void* pair_row, void* tiles,
                                  void* row_w, void* wts, int T, int E, int experts, int top, int max_tiles, int score, int norm_topk, cudaStream_t st) {
  DGPP_REQUIRE(score >= 0 && score <= 2 && (!correction || score < 2), "moe_route_small: score %d", score);
  DGPP_REQUIRE(E >= 1 && E <= kSmallExperts && top >= 1 && top <= kSmallTop && top <= E, "moe_route_small: %d of %d experts", top, E);
  DGPP_REQUIRE(experts >= 1 && experts <= E && (experts == E || wts), "moe_route_small: %d of %d outputs with matrices", experts, E);
  DGPP_REQUIRE(T <= kSmallTokens && max_tiles >= (experts < T * top ? experts : T * top), "moe_route_small: %d tokens in %d tiles", T, max_tiles);
  if (T == 0) return 0;
  const RouteSmall a = {static_cast<const float*>(logits), stride, static_cast<int32_t*>(pair_row), static_cast<int32_t*>(tiles),
                        static_cast<float*>(row_w), static_cast<float*>(wts), static_cast<const float*>(bias),
                        static_cast<const float*>(correction), T, E, top, max_tiles, score, experts, norm_topk};
  moe_route_small_kernel<<<1, kSmallThreads, 0, st>>>(a);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

// x [T, cols] -> xs [tiles * bn, cols], row_w [tiles * bn]: pair (t, j) goes to row pair_row[t * top + j] (negative: nowhere).
DGPP_API int dgpp_moe_scatter_rows(const void* x, const void* pair_row, const void* weights, void* xs, void* row_w, int T, int cols, int top,
                                   int f32, cudaStream_t st) {
  DGPP_REQUIRE(cols % 8 == 0, "moe_scatter_rows: %d columns (a multiple of 8)", cols);
  if (T == 0) return 0;
  const int32_t* pr = static_cast<const int32_t*>(pair_row);
  const float* w = static_cast<const float*>(weights);
  if (f32) moe_scatter_rows_kernel<float><<<T * top, 128, 0, st>>>(static_cast<const float*>(x), pr, w, static_cast<float*>(xs), static_cast<float*>(row_w), cols, top);
  else moe_scatter_rows_kernel<bf16><<<T * top, 128, 0, st>>>(static_cast<const bf16*>(x), pr, w, static_cast<bf16*>(xs), static_cast<float*>(row_w), cols, top);
  DGPP_CUDA_OK(cudaGetLastError());
  return 0;
}

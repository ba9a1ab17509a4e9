// Mixture-of-experts routing that does not depend on the element type of the experts (part of both libraries): scoring and top-k
// of given router logits, and the route plan of a batch (per-expert row ranges + tile map of the grouped products).
//
// Reference counterparts: moe.cu (moe_topk_kernel and its specialisations, count_experts / scan_expert_counts /
// fill_tile_experts / scatter_routes).
#include "moe_route.cuh"

#include <cfloat>

namespace mfq {

// Scoring and top-k with one WARP per token (logits precomputed, E <= 1024, no group limiting): a lane keeps E / 32
// scores in registers, every selection round is a register scan plus five shuffles, and nothing synchronises a block.
__global__ void __launch_bounds__(128) moe_router_topk_warp_kernel(const RouterParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (t >= p.T) return;
  constexpr int kMaxPer = 32;
  const int per = (p.E + 31) >> 5;
  float sc[kMaxPer], sel[kMaxPer];
  float mx = -FLT_MAX;
#pragma unroll
  for (int i = 0; i < kMaxPer; ++i) {
    const int e = i * 32 + lane;
    sc[i] = (i < per && e < p.E) ? p.logits[size_t(t) * p.E + e] : -FLT_MAX;
    mx = fmaxf(mx, sc[i]);
  }
  if (p.sigmoid) {
#pragma unroll
    for (int i = 0; i < kMaxPer; ++i)
      if (i < per) sc[i] = sc[i] == -FLT_MAX ? -FLT_MAX : 1.f / (1.f + __expf(-sc[i]));
  } else {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxPer; ++i)
      if (i < per) {
        const float v = sc[i] == -FLT_MAX ? 0.f : __expf(sc[i] - mx);
        sc[i] = v;
        sum += v;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    const float inv = 1.f / sum;
#pragma unroll
    for (int i = 0; i < kMaxPer; ++i)
      if (i < per) sc[i] = (i * 32 + lane < p.E) ? sc[i] * inv : -FLT_MAX;
  }
#pragma unroll
  for (int i = 0; i < kMaxPer; ++i) {
    const int e = i * 32 + lane;
    const bool live = i < per && e < p.E;
    sel[i] = live ? sc[i] + (p.bias ? p.bias[e] : 0.f) : -FLT_MAX;
    if (live && p.scores_out) p.scores_out[size_t(t) * p.E + e] = sc[i];
  }
  float wsum = 0.f, my_w = 0.f;
  int my_id = 0;
  for (int k = 0; k < p.K; ++k) {
    float best = -FLT_MAX, best_w = 0.f;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < kMaxPer; ++i)
      if (i < per && sel[i] > best) { best = sel[i]; bi = i * 32 + lane; best_w = sc[i]; }  // ascending i: lowest index wins ties
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o), ow = __shfl_xor_sync(0xffffffffu, best_w, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; best_w = ow; }
    }
    if (lane == k) { my_id = bi; my_w = best_w; }
    wsum += best_w;
#pragma unroll
    for (int i = 0; i < kMaxPer; ++i)
      if (i == (bi >> 5) && lane == (bi & 31)) sel[i] = -FLT_MAX;
  }
  if (lane < p.K) {
    const float mul = (p.norm_topk ? 1.f / fmaxf(wsum, 1e-20f) : 1.f) * p.scale;
    p.topk_ids[size_t(t) * p.K + lane] = my_id;
    p.topk_w[size_t(t) * p.K + lane] = my_w * mul;
  }
}

// Route plan for the experts [e_lo, e_hi) owned by this rank (one CTA).  Row order inside an expert depends on atomic
// arrival order; results do not, because each row is computed independently and the un-permute sums a token's K
// contributions in slot order.
//   offsets[e - e_lo]   first sorted row of local expert e (offsets[n_local] = total rows)
//   dest[t*K + k]       sorted row of that (token, slot) pair, -1 if its expert lives on another rank
//   src_token[row]      token of the sorted row
//   tile_map[i]         (local expert, token tile inside it) for the grouped GEMM; padded with (-1, -1)
__global__ void __launch_bounds__(1024) moe_plan_kernel(const int* __restrict__ topk_ids, int entries, int K, int e_lo,
                                                        int e_hi, int token_tile, int* __restrict__ offsets,
                                                        int* __restrict__ dest, int* __restrict__ src_token,
                                                        int2* __restrict__ tile_map, int map_cap,
                                                        int* __restrict__ totals) {
  pdl_trigger();
  pdl_wait();
  __shared__ int cnt[kMaxExperts + 1];
  __shared__ int fill[kMaxExperts];
  __shared__ int tbase[kMaxExperts + 1];
  const int n_local = e_hi - e_lo;
  for (int e = threadIdx.x; e <= n_local; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < entries; i += blockDim.x) {
    const int e = topk_ids[i] - e_lo;
    if (e >= 0 && e < n_local) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  {
    // exclusive prefix sums of the per-expert row and tile counts: one expert per thread, warp scans, then a scan of
    // the 32 warp totals (the block has 1024 threads and at most 512 experts)
    __shared__ int wrow[32], wtile[32];
    const int e = threadIdx.x, lane = e & 31, warp = e >> 5;
    const int c = e < n_local ? cnt[e] : 0;
    const int tl = (c + token_tile - 1) / token_tile;
    int ir = c, it = tl;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int ur = __shfl_up_sync(0xffffffffu, ir, o), ut = __shfl_up_sync(0xffffffffu, it, o);
      if (lane >= o) { ir += ur; it += ut; }
    }
    if (lane == 31) { wrow[warp] = ir; wtile[warp] = it; }
    __syncthreads();
    if (warp == 0) {
      int vr = wrow[lane], vt = wtile[lane];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int ur = __shfl_up_sync(0xffffffffu, vr, o), ut = __shfl_up_sync(0xffffffffu, vt, o);
        if (lane >= o) { vr += ur; vt += ut; }
      }
      wrow[lane] = vr;
      wtile[lane] = vt;
    }
    __syncthreads();
    const int base_r = warp ? wrow[warp - 1] : 0, base_t = warp ? wtile[warp - 1] : 0;
    if (e < n_local) {
      offsets[e] = base_r + ir - c;
      fill[e] = base_r + ir - c;
      tbase[e] = base_t + it - tl;
    }
    if (e == n_local) {  // totals: everything before this (empty) slot
      offsets[n_local] = base_r + ir;
      tbase[n_local] = base_t + it;
      totals[0] = base_r + ir;
      totals[1] = base_t + it;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < entries; i += blockDim.x) {
    const int e = topk_ids[i] - e_lo;
    int row = -1;
    if (e >= 0 && e < n_local) {
      row = atomicAdd(&fill[e], 1);
      src_token[row] = i / K;
    }
    dest[i] = row;
  }
  for (int e = threadIdx.x; e < n_local; e += blockDim.x) {
    const int n = tbase[e + 1] - tbase[e];
    for (int j = 0; j < n; ++j)
      if (tbase[e] + j < map_cap) tile_map[tbase[e] + j] = make_int2(e, j);
  }
  __syncthreads();
  for (int i = tbase[n_local] + threadIdx.x; i < map_cap; i += blockDim.x) tile_map[i] = make_int2(-1, -1);
}

int launch_router_topk_warp(const RouterParams& p, cudaStream_t stream) {
  launch_kernel(moe_router_topk_warp_kernel, dim3((p.T + 3) / 4), dim3(128), 0, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace mfq

using namespace mfq;

// logits [T, E] fp32; the rest as RouterParams
extern "C" int mfq_moe_topk(const float* logits, const float* bias, int* topk_ids, float* topk_w, int T, int E, int K, int sigmoid,
                            int norm_topk, float scale, cudaStream_t stream) {
  if (T <= 0 || E <= 0 || E > kMaxExperts || K <= 0 || K > kMaxTopK || K > E) return -1;
  return launch_router_topk_warp(RouterParams{nullptr, nullptr, bias, topk_ids, topk_w, nullptr, T, 0, E, K, sigmoid, norm_topk, scale, 1, 1,
                                              logits}, stream);
}

extern "C" int mfq_moe_plan(const int* topk_ids, int T, int K, int e_lo, int e_hi, int token_tile, int* offsets, int* dest,
                            int* src_token, void* tile_map, int map_cap, int* totals, cudaStream_t stream) {
  if (e_hi - e_lo > kMaxExperts || e_hi <= e_lo || T <= 0) return -1;
  launch_kernel(moe_plan_kernel, dim3(1), dim3(1024), 0, stream, topk_ids, T * K, K, e_lo, e_hi, token_tile, offsets, dest, src_token,
                                          static_cast<int2*>(tile_map), map_cap, totals);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

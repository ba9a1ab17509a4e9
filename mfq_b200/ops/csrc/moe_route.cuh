// What the routing kernels of every element type share.
#pragma once

#include "common.cuh"

namespace mfq {

constexpr int kMaxExperts = 512;
constexpr int kMaxTopK = 16;

struct RouterParams {
  const __nv_bfloat16* x;      // [T, H]
  const __nv_bfloat16* w;      // [E, H]
  const float* bias;           // [E] selection bias (may be null)
  int* topk_ids;               // [T, K]
  float* topk_w;               // [T, K]
  float* scores_out;           // [T, E] optional (null to skip)
  int T, H, E, K;
  int sigmoid;                 // 0: softmax over experts, 1: sigmoid
  int norm_topk;               // normalise the K selected weights to sum 1
  float scale;                 // multiplier on the final weights (routed scaling factor)
  int n_group, topk_group;     // group-limited routing (n_group <= 1: off)
  const float* logits;         // [T, E] precomputed router logits (null: this kernel computes the dot products)
};

// Scores and picks from given logits, a warp per token (E <= 1024, no group limiting, K <= 32).
int launch_router_topk_warp(const RouterParams& p, cudaStream_t stream);

}  // namespace mfq

// Gated linear attention, shared by its kernels.  Per head, with a [dk, dv] fp32 state S that is carried from token to token:
//   g_t = log2(sigmoid(z_t)) / tau,  or  -log2(e) exp(z_t);   z_t = W_a2 a_t + bias      (a_t: the low-rank projection of the token)
//   S   <- diag(2^g_t) S + k_t v_t^T;   o_t = S^T (q_t scale)
//   y_t = rms_norm(o_t) * w * silu(gate_t)
// With a bonus u (time mixing) the read-out comes before the write and weighs the current token by u instead:
//   o_t = (S + diag(u) k_t v_t^T)^T (q_t scale);   S <- diag(2^g_t) S + k_t v_t^T
// A token's projections lie in one row [q: H dk | k: H dk | v: H dv | gate: H dv | a: rank] (widths as stored, zero padded).
#pragma once

#include "dense_common.cuh"

namespace mfq {

// log2(sigmoid(z)); accurate on both tails
__device__ __forceinline__ float log2_sigmoid(float z) {
  return 1.4426950408889634f * (fminf(z, 0.f) - log1pf(expf(-fabsf(z))));
}
__device__ __forceinline__ float silu_of(float x) { return x / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ float to_float(T x);
template <>
__device__ __forceinline__ float to_float<float>(float x) { return x; }
template <>
__device__ __forceinline__ float to_float<__nv_bfloat16>(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_float(float x);
template <>
__device__ __forceinline__ float from_float<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float x) { return __float2bfloat16(x); }

enum : int { kGlaSigmoid = 0, kGlaExp = 1 };  // how z becomes a decay
constexpr float kGlaFloor = -100.f;           // log2 of a decay that leaves nothing of an fp32 number

struct GlaShape {
  int H, dk, dv, rank;  // as stored: dk, dv multiples of 16, rank of 8
  int row_stride;       // of the projections
  float scale;          // of q
  float inv_tau, inv_dv, eps;  // inv_dv: 1 / the real value channels
  int decay;                   // kGlaSigmoid or kGlaExp
  int norm_stride;             // between two heads' norm weights (0: shared)
  const float* bonus;          // [H dk] or null
};

__device__ __forceinline__ float gla_log2_decay(const GlaShape& s, float z) {
  return s.decay == kGlaSigmoid ? log2_sigmoid(z) * s.inv_tau : fmaxf(-1.4426950408889634f * expf(z), kGlaFloor);
}

}  // namespace mfq

// State-space recurrence with one decay per head, shared by its kernels.  Per head h (of group h / (H / groups)), with an [N, P] fp32
// state S that is carried from token to token:
//   dt_t = softplus(z_t + dt_bias);   g_t = -rate dt_t log2(e)
//   S   <- 2^g_t S + dt_t B_t x_t^T;  y_t = S^T C_t + skip x_t
// A token's x, B and C lie in one row [x: H P | B: groups N | C: groups N] (widths as stored, zero padded), z in a row of its own.
#pragma once

#include "gla.cuh"

namespace mfq {

struct SsdShape {
  int H, groups, N, P;       // as stored: N, P multiples of 16
  int x_stride, z_stride;    // of the rows
  const float* dt_bias;      // [H]
  const float* rate;         // [H] exp(A_log)
  const float* skip;         // [H]
  const int* starts;         // [B + 1] first token of every portion; null: token b is the portion of sequence b
  const int* slot;           // [B] state slot; < 0: skipped
  float* state;              // [slots, H, N, P]
};

// z > 0: z + log(1 + e^-z); accurate on both tails
__device__ __forceinline__ float ssd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace mfq

// Delta rule with a decay per key channel, shared by its kernels.  Per value head h (key head h / (H / G)), with a [dk, dv] fp32
// state S that is carried from token to token, q and k behind their convolution:
//   qn = q / sqrt(sum q^2 + 1e-6) * dim^-1/2,   kn = k / sqrt(sum k^2 + 1e-6),   beta = sigmoid(b_t)
//   g_t = -rate_h log2(e) softplus(z_t),   z_t = W_a2 a_t + dt_bias            (a_t: the low-rank projection of the token)
//   S <- diag(2^g_t) S;   u = beta (v - S^T kn);   S <- S + kn u^T;   o = S^T qn
//   y = rms_norm(o) * w * sigmoid(gate_t)
// Rows: conv [q: G dk | k: G dk | v: H dv] behind the convolution, side [b: up(H) | a: ra | g: rg] as projected (widths as stored).
#pragma once

#include "gla.cuh"

namespace mfq {

struct DeltaShape {
  int H, G, dk, dv;           // as stored: multiples of 16
  int b_cols, ra, rg;         // columns of b, ranks of the decay and gate projections (multiples of 8)
  int conv_stride, side_stride;
  float scale, inv_dv, eps;   // scale: of qn
};

__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float delta_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

}  // namespace mfq

// Score transform of windowed attention, shared by its kernels.  A raw dot product s becomes, in log2 units,
//     c(s) = log2(e) * cap * tanh(s * scale / cap)          (cap > 0)
//     c(s) = log2(e) * s * scale                            (no cap)
// so that a weight is exp2(c(s) - max c).  tanh is odd and increasing: the maximum may be taken over raw scores (scale > 0).
#pragma once

#include "dense_common.cuh"

namespace mfq {

struct ScoreCap {
  float scale_log2;  // scale * log2(e)
  float in;          // 2 * log2(e) * scale / cap: exponent of the exp2 form of tanh
  float out;         // cap * log2(e)
  float small;       // |s| up to this: the series below is exact to fp32 (infinity without a cap)
  float c[5];        // c(s) = s * (c0 + s^2 (c1 + s^2 (c2 + s^2 (c3 + s^2 c4)))): Taylor series of tanh to the 9th power
};

inline ScoreCap make_score_cap(float scale, float cap) {
  const double log2e = 1.4426950408889634;
  ScoreCap k{};
  k.scale_log2 = float(scale * log2e);
  if (cap <= 0.f) {
    k.small = INFINITY;
    k.c[0] = k.scale_log2;
    return k;
  }
  const double r = double(scale) / cap;
  const double series[5] = {1.0, -1.0 / 3, 2.0 / 15, -17.0 / 315, 62.0 / 2835};
  double f = log2e * cap * r;
  for (int i = 0; i < 5; ++i, f *= r * r) k.c[i] = float(f * series[i]);
  k.in = float(2 * log2e * r);
  k.out = float(log2e * cap);
  k.small = float(0.3 / r);  // next term: 0.009 * 0.3^10 = 5e-8 of the result
  return k;
}

__device__ __forceinline__ float window_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float score_small(const ScoreCap& k, float s) {
  const float t = s * s;
  return s * fmaf(t, fmaf(t, fmaf(t, fmaf(t, k.c[4], k.c[3]), k.c[2]), k.c[1]), k.c[0]);
}
// tanh y = 1 - 2 / (exp(2 y) + 1); the absolute error is a few units of 2^-24 times the cap
__device__ __forceinline__ float score_large(const ScoreCap& k, float s) {
  return k.out - k.out * __fdividef(2.f, window_exp2(s * k.in) + 1.f);
}
__device__ __forceinline__ float score_any(const ScoreCap& k, float s) {
  return fabsf(s) <= k.small ? score_small(k, s) : score_large(k, s);
}

// What a head adds to its softmax, in natural units: a score bias by distance, bias[h][min(distance, last)], added to the capped
// score, and one more term exp(sink[h]) of the denominator.
struct ScoreExtra {
  const float* bias;  // [Hq][last + 1] or null
  const float* top;   // [Hq] largest bias of the head (prefill kernel)
  const float* sink;  // [Hq] or null
  int last;
};
constexpr float kLog2e = 1.4426950408889634f;

// First key that a query at position i sees (kept first keys aside): those of its window, or with chunk > 0 those of its chunk
// [n chunk, (n + 1) chunk) of the sequence.
__device__ __forceinline__ int first_key(int i, int window, int chunk) { return chunk > 0 ? i / chunk * chunk : max(0, i - window + 1); }

// Values that carry a rotation by their position: outputs turn back by the query's.  Channel i goes with channel i + half.
struct ValueTurn {
  const float2* rope;  // [rows][half] (cos, sin), or null
  int half, rows;
};

}  // namespace mfq

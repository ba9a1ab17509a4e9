// Stages between the normalised stream and the projections or recurrences of a layer, for activations in bf16 or fp32.
//
//   layer_norm_out    h = (x - mean) / sqrt(var + eps) * w + b of the fp32 stream
//   token_shift       every stream s of a token reads  h + (h' - h) * mu_s,  h' the row of the previous token (zeros before the
//                     first); the last row of a sequence is kept in its state slot
//   short_conv        causal convolution over time per channel (with an optional bias), then SiLU; the last taps - 1 inputs are kept
//                     in the state slot
//   norm_conv         g = h + conv(h) with h = rms_norm(x) * w of the fp32 stream and a causal convolution over time per channel; the
//                     last taps - 1 rows h are kept in the state slot
//
// Batches are ragged: sequence b owns rows starts[b] .. starts[b + 1] - 1 (starts null: row b) and state slot slot[b] (< 0: the
// sequence is skipped).
#include "dense_common.cuh"

namespace mfq {

constexpr int kMixVecs = 4;  // 8-wide vectors a thread keeps in registers

template <typename T>
__global__ void __launch_bounds__(512)
layer_norm_out_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias, T* __restrict__ out, int W,
                      int width, float eps) {
  pdl_trigger();
  __shared__ float red[33];
  const size_t row = blockIdx.x;
  const int nvec = W / 8;
  pdl_wait();
  float v[kMixVecs][8];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kMixVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      load8<float>(x + row * W + vi * 8, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[i][j];  // padding columns are zeros
    }
  }
  const float inv = 1.f / float(width), mean = dense_block_sum(s, red) * inv;
  __syncthreads();
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kMixVecs; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c + j < width) {
        v[i][j] -= mean;
        ss += v[i][j] * v[i][j];
      }
    }
  }
  const float rstd = rsqrtf(dense_block_sum(ss, red) * inv + eps);
#pragma unroll
  for (int i = 0; i < kMixVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      float ww[8], bb[8];
      load8<float>(w + vi * 8, ww);
      load8<float>(bias + vi * 8, bb);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = fmaf(v[i][j] * rstd, ww[j], bb[j]);
      store8<T>(out + row * W + vi * 8, v[i]);
    }
  }
}

// h [T, W]; mu [streams, W]; out [T, streams * W]; last [slots, W] fp32.  The CTA of a sequence's first row reads the kept row and
// replaces it, element by element in the same thread.
template <typename T>
__global__ void __launch_bounds__(256)
token_shift_kernel(const T* __restrict__ h, const float* __restrict__ mu, float* __restrict__ last, const int* __restrict__ slot,
                   const int* __restrict__ starts, const int* __restrict__ tok_seq, T* __restrict__ out, int W, int streams) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, b = tok_seq ? tok_seq[t] : t, s = slot[b];
  const int t0 = starts ? starts[b] : t, t1 = starts ? starts[b + 1] : t + 1;
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float x[8], p[8] = {};
    load8<T>(h + size_t(t) * W + c, x);
    if (t > t0) {
      load8<T>(h + size_t(t - 1) * W + c, p);
    } else if (s >= 0) {
      load8<float>(last + size_t(s) * W + c, p);
      float e[8];
      load8<T>(h + size_t(t1 - 1) * W + c, e);
      store8<float>(last + size_t(s) * W + c, e);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) p[j] -= x[j];
    for (int i = 0; i < streams; ++i) {
      float m[8];
      load8<float>(mu + size_t(i) * W + c, m);
#pragma unroll
      for (int j = 0; j < 8; ++j) m[j] = fmaf(p[j], m[j], x[j]);
      store8<T>(out + (size_t(t) * streams + i) * W + c, m);
    }
  }
}

struct ShortConvParams {
  const float* w;     // [taps, C], last row for the current token
  const float* bias;  // [C] or null
  float* state;       // [slots, taps - 1, C], oldest first
  const int* slot;    // [B]
  const int* starts;  // [B + 1] or null
  int C, taps, in_stride, out_stride;
};

// A thread owns 8 channels and a run of consecutive tokens; TAPS is an upper bound of the taps (missing ones weigh nothing).
constexpr int kConvRunTokens = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ x, T* __restrict__ out, const ShortConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, s = p.slot[b], c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (s < 0 || c >= p.C) return;
  const int r0 = p.starts ? p.starts[b] : b, len = p.starts ? p.starts[b + 1] - r0 : 1;
  const int n0 = blockIdx.y * kConvRunTokens, n1 = min(len, n0 + kConvRunTokens), hist = p.taps - 1;
  if (n0 >= len) return;
  float* st = p.state + size_t(s) * hist * p.C + c;
  auto in = [&](int n, float(&v)[8]) {  // input n tokens into the portion; n < 0: the kept ones
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
    if (n >= 0) load8<T>(x + size_t(r0 + n) * p.in_stride + c, v);
    else if (n + hist >= 0) load8<float>(st + size_t(n + hist) * p.C, v);
  };
  float w[TAPS][8], win[TAPS][8], add[8] = {};  // win[i]: input i - (TAPS - 1) tokens from the current one
  if (p.bias) load8<float>(p.bias + c, add);
#pragma unroll
  for (int i = 0; i < TAPS; ++i) {
#pragma unroll
    for (int j = 0; j < 8; ++j) w[i][j] = 0.f;
    if (i - (TAPS - p.taps) >= 0) load8<float>(p.w + size_t(i - (TAPS - p.taps)) * p.C + c, w[i]);
    if (i > 0) in(n0 + i - TAPS, win[i]);
  }
  constexpr int kAhead = 4;  // inputs requested before the first of them is used
  for (int m = n0; m < n1; m += kAhead) {
    float next[kAhead][8];
#pragma unroll
    for (int e = 0; e < kAhead; ++e)
      if (m + e < n1) in(m + e, next[e]);
#pragma unroll
    for (int e = 0; e < kAhead; ++e) {
      if (m + e >= n1) break;
      float y[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
#pragma unroll
        for (int i = 0; i + 1 < TAPS; ++i) win[i][j] = win[i + 1][j];
        win[TAPS - 1][j] = next[e][j];
        float a = add[j];
#pragma unroll
        for (int i = 0; i < TAPS; ++i) a = fmaf(w[i][j], win[i][j], a);
        y[j] = sizeof(T) == 4 ? a / (1.f + expf(-a)) : __fdividef(a, 1.f + __expf(-fmaxf(a, -80.f)));
      }
      store8<T>(out + size_t(r0 + m + e) * p.out_stride + c, y);
    }
  }
  // Portions of one token: this thread is the only one that reads these kept inputs, so it may replace them.
  if (!p.starts) {
#pragma unroll
    for (int i = 1; i < TAPS; ++i)
      if (i - (TAPS - p.taps) >= 1) store8<float>(st + size_t(i - (TAPS - p.taps) - 1) * p.C, win[i]);
  }
}

// The kept inputs after a portion of any length, as a launch of its own (blocks of the convolution still read the old ones).
template <typename T>
__global__ void __launch_bounds__(128)
short_conv_state_kernel(const T* __restrict__ x, const ShortConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, s = p.slot[b], c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (s < 0 || c >= p.C) return;
  const int r0 = p.starts[b], len = p.starts[b + 1] - r0, hist = p.taps - 1;
  float* st = p.state + size_t(s) * hist * p.C + c;
  for (int i = 0; i < hist; ++i) {  // ascending: place i reads place i + len >= i
    const int n = len - hist + i;
    float v[8];
    if (n >= 0) load8<T>(x + size_t(r0 + n) * p.in_stride + c, v);
    else load8<float>(st + size_t(n + hist) * p.C, v);
    store8<float>(st + size_t(i) * p.C, v);
  }
}

template <typename T>
static int launch_short_conv(const void* x, void* out, const ShortConvParams& p, int B, int max_q, cudaStream_t stream) {
  const T* xt = static_cast<const T*>(x);
  T* ot = static_cast<T*>(out);
  const int blocks = (p.C / 8 + 127) / 128;
  const dim3 grid(blocks, (max_q + kConvRunTokens - 1) / kConvRunTokens, B);
  if (p.taps <= 4) launch_kernel(short_conv_kernel<T, 4>, grid, dim3(128), 0, stream, xt, ot, p);
  else launch_kernel(short_conv_kernel<T, 8>, grid, dim3(128), 0, stream, xt, ot, p);
  if (p.starts && p.taps > 1) launch_kernel(short_conv_state_kernel<T>, dim3(blocks, B), dim3(128), 0, stream, xt, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

struct NormConvParams {
  const float* x;       // [T, W] fp32 stream
  const float* norm_w;  // [W]
  const float* w;       // [taps, W], last row for the current token
  float* state;         // [slots, taps - 1, W], oldest first
  const int* slot;      // [B]
  const int* starts;    // [B + 1] or null
  int W, taps;
  float inv_width, eps;
};

// A CTA takes a run of tokens of a sequence: first the root mean squares of its rows and of the taps - 1 before them, then every thread
// walks the run for 4 channels at a time.  The CTA of the sequence's first run is the only one that reads the kept rows, so it also
// replaces them (by the portion's last rows), channel by channel in the same thread.
constexpr int kNormMaxRun = 32, kNormMaxTaps = 8, kNormThreads = 512;
template <typename T, int TAPS>
__global__ void __launch_bounds__(kNormThreads, TAPS <= 4 ? 2 : 1)
norm_conv_kernel(T* __restrict__ out, const NormConvParams p, int run) {
  pdl_trigger();
  pdl_wait();
  constexpr int kRows = kNormMaxRun + 2 * (kNormMaxTaps - 1), kWarps = kNormThreads / 32, kAhead = TAPS <= 4 ? 4 : 8;
  __shared__ float part[kRows * kWarps], scale[kRows];
  const int b = blockIdx.y, s = p.slot[b], W = p.W;
  const int r0 = p.starts ? p.starts[b] : b, len = p.starts ? p.starts[b + 1] - r0 : 1;
  const int n0 = blockIdx.x * run, n1 = min(len, n0 + run), hist = p.taps - 1;
  if (n0 >= len) return;
  const int first = max(0, n0 - hist), tail = n0 == 0 ? max(n1, len - hist) : len;  // rows first .. n1 - 1, then tail .. len - 1
  const int rows = n1 - first + len - tail;
  const float* x = p.x + size_t(r0) * W;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int each = rows <= warps ? warps / rows : 2;  // shares of a row
  for (int j = warp; j < rows * each; j += warps) {
    const int i = j / each, n = i < n1 - first ? first + i : tail + i - (n1 - first);
    const float* row = x + size_t(n) * W;
    float ss = 0.f;
#pragma unroll 8
    for (int c = ((j - i * each) * 32 + lane) * 4; c < W; c += each * 128) {
      const float4 v = *reinterpret_cast<const float4*>(row + c);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) part[j] = ss;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < rows; i += blockDim.x) {
    float ss = 0.f;
    for (int z = 0; z < each; ++z) ss += part[i * each + z];
    scale[i] = rsqrtf(fmaf(ss, p.inv_width, p.eps));
  }
  __syncthreads();
  float* st = s >= 0 && hist > 0 ? p.state + size_t(s) * hist * W : nullptr;
  auto load4 = [](const float* src, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(src);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  };
  for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
    float w[TAPS][4], win[TAPS - 1][4], nw[4];  // win: the rows before the current one, oldest first
    load4(p.norm_w + c, nw);
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      const bool used = i >= TAPS - p.taps;
      const int n = n0 + i - (TAPS - 1);
#pragma unroll
      for (int j = 0; j < 4; ++j) w[i][j] = 0.f;
      if (used) load4(p.w + size_t(i - (TAPS - p.taps)) * W + c, w[i]);
      if (i < TAPS - 1) {
        float f = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) win[i][j] = 0.f;
        if (used && n >= 0) {
          load4(x + size_t(n) * W + c, win[i]);
          f = scale[n - first];
        } else if (used && st) {
          load4(st + size_t(n + hist) * W + c, win[i]);
        }
        if (n >= 0) {
#pragma unroll
          for (int j = 0; j < 4; ++j) win[i][j] *= f * nw[j];
        }
      }
    }
    for (int m = n0; m < n1; m += kAhead) {
      float h[kAhead][4];
#pragma unroll
      for (int e = 0; e < kAhead; ++e)
        if (m + e < n1) load4(x + size_t(m + e) * W + c, h[e]);
#pragma unroll
      for (int e = 0; e < kAhead; ++e) {
        if (m + e < n1) {
          const float f = scale[m + e - first];
          float y[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            h[e][j] *= f * nw[j];
            y[j] = fmaf(w[TAPS - 1][j], h[e][j], h[e][j]);
#pragma unroll
            for (int i = 0; i < TAPS - 1; ++i) y[j] = fmaf(w[i][j], i + e < TAPS - 1 ? win[min(i + e, TAPS - 2)][j] : h[max(i + e - (TAPS - 1), 0)][j], y[j]);
          }
          T* dst = out + size_t(r0 + m + e) * W + c;
          if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1], y[2], y[3]);
          } else {
            __nv_bfloat162 q[2] = {__floats2bfloat162_rn(y[0], y[1]), __floats2bfloat162_rn(y[2], y[3])};
            *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(q);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i)  // a further batch follows a whole one
#pragma unroll
        for (int j = 0; j < 4; ++j) win[i][j] = h[kAhead - (TAPS - 1) + i][j];
    }
    if (n0 == 0 && st) {
      for (int i = 0; i < hist; ++i) {  // ascending: place i reads place i + len > i
        const int n = len - hist + i;
        float v[4];
        if (n >= 0) {
          const float f = scale[n < n1 ? n - first : n1 - first + n - tail];
          load4(x + size_t(n) * W + c, v);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] *= f * nw[j];
        } else {
          load4(st + size_t(n + hist) * W + c, v);
        }
        *reinterpret_cast<float4*>(st + size_t(i) * W + c) = make_float4(v[0], v[1], v[2], v[3]);
      }
    }
  }
}

// One row per sequence, up to 4 taps, 8 VECS channels per thread.
constexpr int kStepTaps = 4;
template <typename T, int VECS>
__global__ void __launch_bounds__(kNormThreads, 1)
norm_conv_step_kernel(T* __restrict__ out, const NormConvParams p) {
  pdl_trigger();
  __shared__ float red[33];
  const int W = p.W, hist = p.taps - 1;
  const size_t b = blockIdx.x;
  float w[VECS][kStepTaps][8], nw[VECS][8], x[VECS][8];
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < W) {
      load8<float>(p.norm_w + c, nw[k]);
#pragma unroll
      for (int i = 0; i < kStepTaps; ++i)
        if (i < p.taps) load8<float>(p.w + size_t(i) * W + c, w[k][i]);
    }
  }
  pdl_wait();
  const int s = p.slot[b];
  float* st = s >= 0 && hist > 0 ? p.state + size_t(s) * hist * W : nullptr;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < W) {
      load8<float>(p.x + b * W + c, x[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(x[k][j], x[k][j], ss);
    }
  }
  float y[VECS][8];
#pragma unroll
  for (int k = 0; k < VECS; ++k) {  // the kept rows, moved up by one
    const int c = (threadIdx.x + k * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) y[k][j] = 0.f;
    if (c < W && st) {
#pragma unroll
      for (int i = 0; i < kStepTaps - 1; ++i) {
        if (i < hist) {
          float v[8];
          load8<float>(st + size_t(i) * W + c, v);
          if (i > 0) store8<float>(st + size_t(i - 1) * W + c, v);
#pragma unroll
          for (int j = 0; j < 8; ++j) y[k][j] = fmaf(w[k][i][j], v[j], y[k][j]);
        }
      }
    }
  }
  const float f = rsqrtf(fmaf(dense_block_sum(ss, red), p.inv_width, p.eps));
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < W) {
      float last[8];
#pragma unroll
      for (int i = 0; i < kStepTaps; ++i)
        if (i == hist) {
#pragma unroll
          for (int j = 0; j < 8; ++j) last[j] = w[k][i][j];
        }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        x[k][j] *= f * nw[k][j];
        y[k][j] = fmaf(last[j], x[k][j], y[k][j]) + x[k][j];
      }
      store8<T>(out + b * W + c, y[k]);
      if (st) store8<float>(st + size_t(hist - 1) * W + c, x[k]);
    }
  }
}

template <typename T>
static int launch_norm_conv(void* out, const NormConvParams& p, int B, int max_q, int tokens, cudaStream_t stream) {
  T* o = static_cast<T*>(out);
  const int vecs = p.W / 8;
  if (!p.starts && p.taps <= kStepTaps && vecs <= 2 * kNormThreads) {
    if (vecs <= kNormThreads) launch_kernel(norm_conv_step_kernel<T, 1>, dim3(B), dim3((vecs + 31) / 32 * 32), 0, stream, o, p);
    else launch_kernel(norm_conv_step_kernel<T, 2>, dim3(B), dim3((vecs / 2 + 31) / 32 * 32), 0, stream, o, p);
    return cudaGetLastError() == cudaSuccess ? 0 : -7;
  }
  const int threads = min(kNormThreads, (p.W / 4 + 31) / 32 * 32);
  const int run = min(kNormMaxRun, max(8, (tokens + 8 * 148 - 1) / (8 * 148) * 4));  // at most a wave of two CTAs per SM, if that many tokens fit
  const dim3 grid((max_q + run - 1) / run, B);
  if (p.taps <= 4) launch_kernel(norm_conv_kernel<T, 4>, grid, dim3(threads), 0, stream, o, p, run);
  else launch_kernel(norm_conv_kernel<T, kNormMaxTaps>, grid, dim3(threads), 0, stream, o, p, run);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace mfq

using namespace mfq;

extern "C" int mfq_layer_norm_out(const float* x, const float* w, const float* bias, void* out, int M, int W, int width, float eps, int fp32,
                                  cudaStream_t stream) {
  if (M <= 0 || W <= 0 || W % 8 || W > 8 * kMixVecs * 512 || width <= 0 || width > W) return -1;
  const int nvec = W / 8;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 256) threads = max(256, ((nvec + kMixVecs - 1) / kMixVecs + 31) / 32 * 32);
  if (fp32) launch_kernel(layer_norm_out_kernel<float>, dim3(M), dim3(threads), 0, stream, x, w, bias, static_cast<float*>(out), W, width, eps);
  else launch_kernel(layer_norm_out_kernel<__nv_bfloat16>, dim3(M), dim3(threads), 0, stream, x, w, bias, static_cast<__nv_bfloat16*>(out), W, width, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

extern "C" int mfq_token_shift(const void* h, const float* mu, float* last, const int* slot, const int* starts, const int* tok_seq, void* out,
                               int T_, int W, int streams, int fp32, cudaStream_t stream) {
  if (T_ <= 0 || W <= 0 || W % 8 || streams <= 0 || (starts && !tok_seq)) return -1;
  const int threads = min(256, (W / 8 + 31) / 32 * 32);
  if (fp32)
    launch_kernel(token_shift_kernel<float>, dim3(T_), dim3(threads), 0, stream, static_cast<const float*>(h), mu, last, slot, starts, tok_seq,
                  static_cast<float*>(out), W, streams);
  else
    launch_kernel(token_shift_kernel<__nv_bfloat16>, dim3(T_), dim3(threads), 0, stream, static_cast<const __nv_bfloat16*>(h), mu, last, slot,
                  starts, tok_seq, static_cast<__nv_bfloat16*>(out), W, streams);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// x [T, W] fp32; out [T, W] = h + conv(h); w [taps, W]; state [slots, taps - 1, W]; starts null: row b belongs to
// sequence b; tokens: rows of all portions
extern "C" int mfq_norm_conv(const float* x, const float* norm_w, const float* w, float* state, const int* slot, const int* starts, void* out,
                             int B, int max_q, int tokens, int W, int width, int taps, float eps, int fp32, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || max_q <= 0 || tokens <= 0 || W <= 0 || W % 8 || width <= 0 || width > W || taps < 1 || taps > kNormMaxTaps) return -1;
  if (taps > 1 && !state) return -1;
  const NormConvParams p{x, norm_w, w, state, slot, starts, W, taps, 1.f / float(width), eps};
  return fp32 ? launch_norm_conv<float>(out, p, B, starts ? max_q : 1, tokens, stream)
              : launch_norm_conv<__nv_bfloat16>(out, p, B, starts ? max_q : 1, tokens, stream);
}

// x: rows of in_stride, channels 0 .. C - 1; w [taps, C]; bias [C] or null; state [slots, taps - 1, C]; starts null: row b belongs to sequence b
extern "C" int mfq_short_conv(const void* x, int in_stride, const float* w, const float* bias, float* state, const int* slot, const int* starts, void* out,
                              int out_stride, int B, int max_q, int C, int taps, int fp32, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || max_q <= 0 || C <= 0 || C % 8 || taps < 1 || taps > 8 || in_stride % 8 || out_stride % 8) return -1;
  const ShortConvParams p{w, bias, state, slot, starts, C, taps, in_stride, out_stride};
  return fp32 ? launch_short_conv<float>(x, out, p, B, starts ? max_q : 1, stream)
              : launch_short_conv<__nv_bfloat16>(x, out, p, B, starts ? max_q : 1, stream);
}

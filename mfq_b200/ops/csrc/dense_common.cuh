// Shared pieces of the unquantized (bf16 or fp32) model path: 8-wide vector access, reductions, and the output stage of
// the dense products.  Every width of this path is stored rounded up to a multiple of 8 or 16 with zeros, so 16-byte
// accesses are always aligned and never need a tail.
#pragma once

#include "common.cuh"

namespace mfq {

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <>
__device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <>
__device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 o;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = o;
}

// Block-wide sum over <= 1024 threads; `red` is 33 floats of shared memory.
__device__ __forceinline__ float dense_block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float x = lane < nw ? red[lane] : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
    if (lane == 0) red[32] = x;
  }
  __syncthreads();
  return red[32];
}

// What happens to a product row before it is stored.
enum : int {
  kDenseBias = 0,   // out[t, n] = v + bias[n]
  kDenseGlu = 1,    // weight rows packed in blocks of 16 = 8 gate rows | 8 up rows: out = clipped GLU, half as wide
  kDenseGelu = 2,   // out[t, n] = gelu_tanh(v + bias[n]) * table[ids[t], n]
  kDenseGeluGlu = 3,  // rows packed as for kDenseGlu: out = gelu_tanh(gate) * up, half as wide
  kDenseSoftcap = 4,  // out[t, n] = limit * tanh((v + bias[n]) / limit)
  kDenseAdd = 5,      // x[t, n] += alpha * (v + bias[n]) on the fp32 stream x = out
  kDenseReluGlu = 6,  // rows packed as for kDenseGlu: out = max(gate, 0) * up, half as wide
  kDenseSiluGlu = 7,  // ... out = silu(gate) * up
  kDenseFloat = 8,    // fp32 out[t, n] = v + bias[n]
  kDenseRelu2 = 9,    // out[t, n] = max(v + bias[n], 0)^2
};
__host__ __device__ constexpr bool dense_is_glu(int kind) {
  return kind == kDenseGlu || kind == kDenseGeluGlu || kind == kDenseReluGlu || kind == kDenseSiluGlu;
}

struct DenseEpilogue {
  int kind;
  const float* bias;  // [N] or null
  float alpha, limit;  // GLU: y = g sigmoid(alpha g) (u + 1), g = min(gate, limit), u = clamp(up, -limit, limit); soft cap: limit; add: alpha
  const void* table;   // GELU: [tokens of the vocabulary, N] in the activation type
  const int* ids;
  void* out;
  int ldo;
};

__device__ __forceinline__ float clipped_glu(float gate, float up, float alpha, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float gated_unit(const DenseEpilogue& e, float gate, float up) {
  switch (e.kind) {
    case kDenseGlu: return clipped_glu(gate, up, e.alpha, e.limit);
    case kDenseGeluGlu: return gelu_tanh(gate) * up;
    case kDenseReluGlu: return fmaxf(gate, 0.f) * up;
    default: return gate / (1.f + expf(-gate)) * up;
  }
}

// One output item of token `t`: 8 packed rows from `n0`, or 16 for the GLU kinds.  `load(n, v)` fetches the finished fp32 sums
// of rows n .. n + 7.
template <typename T, typename Load>
__device__ __forceinline__ void dense_store_item(const DenseEpilogue& e, int t, int n0, Load&& load) {
  float v[8];
  load(n0, v);
  if (e.bias) {
    float b[8];
    load8<float>(e.bias + n0, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] += b[i];
  }
  if (e.kind == kDenseAdd) {
    float* x = static_cast<float*>(e.out) + size_t(t) * e.ldo + n0;
    float r[8];
    load8<float>(x, r);
#pragma unroll
    for (int i = 0; i < 8; ++i) r[i] = fmaf(e.alpha, v[i], r[i]);
    store8<float>(x, r);
    return;
  }
  if (e.kind == kDenseFloat) {
    store8<float>(static_cast<float*>(e.out) + size_t(t) * e.ldo + n0, v);
    return;
  }
  T* out = static_cast<T*>(e.out) + size_t(t) * e.ldo;
  if (dense_is_glu(e.kind)) {
    float u[8];
    load(n0 + 8, u);
    if (e.bias) {
      float b[8];
      load8<float>(e.bias + n0 + 8, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) u[i] += b[i];
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = gated_unit(e, v[i], u[i]);
    store8<T>(out + (n0 >> 1), v);
    return;
  }
  if (e.kind == kDenseGelu) {
    float g[8];
    load8<T>(static_cast<const T*>(e.table) + size_t(e.ids[t]) * e.ldo + n0, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = gelu_tanh(v[i]) * g[i];
  }
  if (e.kind == kDenseRelu2) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = fmaxf(v[i], 0.f) * fmaxf(v[i], 0.f);
  }
  if (e.kind == kDenseSoftcap) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = e.limit * tanhf(v[i] / e.limit);
  }
  store8<T>(out + n0, v);
}

}  // namespace mfq

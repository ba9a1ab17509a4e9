// Row movement around the expert products of the unquantized path (dense_gemm.cu, expert form; routing in moe_route.cu).
//
//   moe_rows_sorted   copy of activation rows in expert order
//   moe_add_experts   x[t] += scale * sum_k w[t, k] * y[dest[t, k]]  on the fp32 stream
#include "dense_common.cuh"

namespace mfq {

__global__ void __launch_bounds__(256)
moe_rows_sorted_kernel(const uint4* __restrict__ x, const int* __restrict__ src, const int* __restrict__ totals, uint4* __restrict__ out,
                       int vecs, int stride) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  if (row >= totals[0]) return;
  const uint4* from = x + size_t(src[row]) * stride;
  for (int i = threadIdx.x; i < vecs; i += blockDim.x) out[size_t(row) * vecs + i] = from[i];
}

template <typename T>
__global__ void __launch_bounds__(256)
moe_add_experts_kernel(const T* __restrict__ y, const int* __restrict__ dest, const float* __restrict__ weight, float* __restrict__ x, int W,
                       int K, float scale) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float acc[8] = {}, r[8];
    for (int k = 0; k < K; ++k) {
      const int row = dest[size_t(t) * K + k];
      if (row < 0) continue;
      const float w = weight[size_t(t) * K + k];
      load8<T>(y + size_t(row) * W + c, r);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = fmaf(w, r[j], acc[j]);
    }
    load8<float>(x + size_t(t) * W + c, r);
#pragma unroll
    for (int j = 0; j < 8; ++j) r[j] = fmaf(scale, acc[j], r[j]);
    store8<float>(x + size_t(t) * W + c, r);
  }
}

}  // namespace mfq

using namespace mfq;

// Rows of `bytes` (a multiple of 16), `stride` bytes apart in x and packed in out.
extern "C" int mfq_moe_rows_sorted(const void* x, const int* src, const int* totals, void* out, int max_rows, int bytes, int stride,
                                   cudaStream_t stream) {
  if (max_rows <= 0 || bytes <= 0 || bytes % 16 || stride % 16) return -1;
  launch_kernel(moe_rows_sorted_kernel, dim3(max_rows), dim3(min(256, (bytes / 16 + 31) / 32 * 32)), 0, stream, static_cast<const uint4*>(x),
                src, totals, static_cast<uint4*>(out), bytes / 16, stride / 16);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

extern "C" int mfq_moe_add_experts(const void* y, const int* dest, const float* weight, float* x, int T_, int W, int K, float scale, int fp32,
                                   cudaStream_t stream) {
  if (T_ <= 0 || W <= 0 || W % 8 || K <= 0) return -1;
  const dim3 block(min(256, (W / 8 + 31) / 32 * 32));
  if (fp32) launch_kernel(moe_add_experts_kernel<float>, dim3(T_), block, 0, stream, static_cast<const float*>(y), dest, weight, x, W, K, scale);
  else launch_kernel(moe_add_experts_kernel<__nv_bfloat16>, dim3(T_), block, 0, stream, static_cast<const __nv_bfloat16*>(y), dest, weight, x, W, K, scale);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

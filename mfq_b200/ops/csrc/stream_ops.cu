// fp32 residual stream of a decoder whose sublayers are normalised on their OUTPUT, and the per-head stage between the
// q/k/v projection and attention, for activations in bf16 or fp32.
//
//   embed_scaled      x = table[id] * scale              -> fp32 stream + copy in the activation type
//   norm_add          x += rms_norm(y) * w               -> fp32 stream + copy in the activation type, one pass over y and x
//   norm_out          h = rms_norm(x) * w                -> activation type (input of the LM head)
//   qkv_finish        per head: RMS norm of q and k, rotation of the leading channels, blending of v with the values another
//                     layer computed for the same token, K / V into their pages
//
// "rms_norm" divides by sqrt(mean(x^2) + eps) over the model's true width; weights arrive in fp32 in the form they multiply
// with.  Padding columns hold zeros and stay zero because their weights are zero.
#include "dense_common.cuh"

namespace mfq {

constexpr int kStreamVecs = 4;  // 8-wide vectors a thread keeps in registers (rows up to 8 * 4 * 512 wide)

template <typename T>
__global__ void embed_scaled_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale, float* __restrict__ x,
                                    T* __restrict__ xa, int W) {
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x, src = size_t(ids[row]);
  for (int i = threadIdx.x; i < W / 8; i += blockDim.x) {
    float v[8];
    load8<T>(table + src * W + i * 8, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= scale;
    store8<float>(x + row * W + i * 8, v);
    if (xa) store8<T>(xa + row * W + i * 8, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(512)
norm_add_kernel(const T* __restrict__ y, const float* __restrict__ w, float* __restrict__ x, T* __restrict__ xa, int W,
                float inv_width, float eps) {
  pdl_trigger();
  __shared__ float red[33];
  const size_t row = blockIdx.x;
  const int nvec = W / 8;
  pdl_wait();
  float v[kStreamVecs][8], r[kStreamVecs][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kStreamVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      load8<T>(y + row * W + vi * 8, v[i]);
      load8<float>(x + row * W + vi * 8, r[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[i][j] * v[i][j];
    }
  }
  const float rstd = rsqrtf(dense_block_sum(ss, red) * inv_width + eps);
#pragma unroll
  for (int i = 0; i < kStreamVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      float ww[8];
      load8<float>(w + vi * 8, ww);
#pragma unroll
      for (int j = 0; j < 8; ++j) r[i][j] += v[i][j] * rstd * ww[j];
      store8<float>(x + row * W + vi * 8, r[i]);
      if (xa) store8<T>(xa + row * W + vi * 8, r[i]);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(512)
norm_out_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ out, int W, float inv_width, float eps) {
  pdl_trigger();
  __shared__ float red[33];
  const size_t row = blockIdx.x;
  const int nvec = W / 8;
  pdl_wait();
  float v[kStreamVecs][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kStreamVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      load8<float>(x + row * W + vi * 8, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[i][j] * v[i][j];
    }
  }
  const float rstd = rsqrtf(dense_block_sum(ss, red) * inv_width + eps);
#pragma unroll
  for (int i = 0; i < kStreamVecs; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      float ww[8];
      load8<float>(w + vi * 8, ww);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= rstd * ww[j];
      store8<T>(out + row * W + vi * 8, v[i]);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// qkv rows [Hq * dk | Hk * dk | Hk * dv] (dk, dv: head widths as stored, multiples of 16; d: the true q / k width the norm
// averages over).  `L` lanes (a power of two) share a head, 8 channels each; a warp takes 32 / L heads of one token.
// The rotation reads (cos, sin) of the token's position from a table [positions][rot / 2] and its partner channel from
// shared memory.  Pages: K [page][Hk][16][dk], V [page][Hk][16][dv]; slot < 0: the token is not cached.
// ---------------------------------------------------------------------------------------------
struct QkvFinishParams {
  int T, Hq, Hk, d, dk, dv, rot, row_stride, page_size, L, table_rows;
  float eps, lambda;        // lambda: share of the other layer's values
  int first_stride;         // row stride of `v_first`
  const float* q_norm;
  const float* k_norm;      // [dk] fp32 or null: no norm
  const float2* rope;       // (cos, sin)
  const int* positions;
  const int* slots;
};

template <typename T>
__global__ void __launch_bounds__(256)
qkv_finish_kernel(const T* __restrict__ qkv, const T* __restrict__ v_first, T* __restrict__ q_out, T* __restrict__ k_pages,
                  T* __restrict__ v_pages, const QkvFinishParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float sh[8][32 * 8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_warp = 32 / p.L, sub = lane / p.L, c = lane - sub * p.L;  // c: my 8-channel chunk
  const int heads = p.Hq + 2 * p.Hk;
  const int groups = (heads + per_warp - 1) / per_warp;  // head groups of a token
  const int gw = blockIdx.x * 8 + warp;
  if (gw >= p.T * groups) return;  // whole warps leave together
  const int t = gw / groups, h = (gw - t * groups) * per_warp + sub;
  const bool live_head = h < heads;
  const bool is_q = h < p.Hq, is_v = h >= p.Hq + p.Hk;
  const int width = is_v ? p.dv : p.dk;
  const bool mine = live_head && c * 8 < width;
  const T* row = qkv + size_t(t) * p.row_stride;
  const int col = is_v ? (p.Hq + p.Hk) * p.dk + (h - p.Hq - p.Hk) * p.dv : h * p.dk;
  float v[8];
  if (mine) {
    load8<T>(row + col + c * 8, v);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
  }
  const float* nw = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
  for (int o = p.L >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (mine && nw) {
    const float inv = rsqrtf(ss / float(p.d) + p.eps);
    float ww[8];
    load8<float>(nw + c * 8, ww);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= inv * ww[j];
  }
  float* mysh = sh[warp] + sub * p.L * 8;
#pragma unroll
  for (int j = 0; j < 8; ++j) mysh[c * 8 + j] = v[j];
  __syncwarp();
  if (!mine) return;
  if (!is_v && c * 8 < p.rot) {
    const int half = p.rot >> 1, pos = min(p.positions[t], p.table_rows - 1);
    const float2* tab = p.rope + size_t(pos) * half;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = c * 8 + j;
      if (i < half) {
        const float2 cs = tab[i];
        v[j] = v[j] * cs.x - mysh[i + half] * cs.y;
      } else if (i < p.rot) {
        const float2 cs = tab[i - half];
        v[j] = v[j] * cs.x + mysh[i - half] * cs.y;
      }
    }
  }
  if (is_q) {
    store8<T>(q_out + (size_t(t) * p.Hq + h) * p.dk + c * 8, v);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const int page = slot / p.page_size, off = slot - page * p.page_size;
  if (!is_v) {
    store8<T>(k_pages + ((size_t(page) * p.Hk + (h - p.Hq)) * p.page_size + off) * p.dk + c * 8, v);
    return;
  }
  const int g = h - p.Hq - p.Hk;
  if (v_first) {
    float f[8];
    load8<T>(v_first + size_t(t) * p.first_stride + g * p.dv + c * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = (1.f - p.lambda) * v[j] + p.lambda * f[j];
  }
  store8<T>(v_pages + ((size_t(page) * p.Hk + g) * p.page_size + off) * p.dv + c * 8, v);
}

static int stream_threads(int W) {
  const int nvec = W / 8;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 256) threads = max(256, ((nvec + kStreamVecs - 1) / kStreamVecs + 31) / 32 * 32);
  return threads <= 512 ? threads : -1;
}

}  // namespace mfq

using namespace mfq;

#define MFQ_BY_TYPE(fp32, CALL)                       \
  do {                                                \
    if (fp32) { using T = float; CALL; }              \
    else { using T = __nv_bfloat16; CALL; }           \
  } while (0)

// table [V, W]; x [T, W] fp32; xa [T, W] (may be null: fp32 activations are the stream itself)
extern "C" int mfq_embed_scaled(const int* ids, const void* table, float scale, float* x, void* xa, int T_, int W, int fp32,
                                cudaStream_t stream) {
  if (T_ <= 0 || W <= 0 || W % 8) return -1;
  const int threads = min(256, (W / 8 + 31) / 32 * 32);
  MFQ_BY_TYPE(fp32, launch_kernel(embed_scaled_kernel<T>, dim3(T_), dim3(threads), 0, stream, ids, static_cast<const T*>(table), scale,
                                  x, static_cast<T*>(xa), W));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// x += y / sqrt(mean(y^2) + eps) * w over rows of `W` stored columns, `width` of which are real
extern "C" int mfq_norm_add(const void* y, const float* w, float* x, void* xa, int M, int W, int width, float eps, int fp32,
                            cudaStream_t stream) {
  const int threads = W > 0 && W % 8 == 0 ? stream_threads(W) : -1;
  if (M <= 0 || threads < 0 || width <= 0 || width > W) return -1;
  MFQ_BY_TYPE(fp32, launch_kernel(norm_add_kernel<T>, dim3(M), dim3(threads), 0, stream, static_cast<const T*>(y), w, x,
                                  static_cast<T*>(xa), W, 1.f / float(width), eps));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

extern "C" int mfq_norm_out(const float* x, const float* w, void* out, int M, int W, int width, float eps, int fp32,
                            cudaStream_t stream) {
  const int threads = W > 0 && W % 8 == 0 ? stream_threads(W) : -1;
  if (M <= 0 || threads < 0 || width <= 0 || width > W) return -1;
  MFQ_BY_TYPE(fp32, launch_kernel(norm_out_kernel<T>, dim3(M), dim3(threads), 0, stream, x, w, static_cast<T*>(out), W,
                                  1.f / float(width), eps));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

extern "C" int mfq_qkv_finish(const void* qkv, int row_stride, const void* v_first, int first_stride, float lambda, void* q_out,
                              void* k_pages, void* v_pages, const int* positions, const int* slots, const float* q_norm,
                              const float* k_norm, const float* rope, int table_rows, int T_, int Hq, int Hk, int d, int dk, int dv,
                              int rot, int page_size, float eps, int fp32, cudaStream_t stream) {
  if (T_ <= 0 || Hq <= 0 || Hk <= 0 || Hq % Hk || dk % 16 || dv % 16 || dk > 256 || dv > 256 || d <= 0 || d > dk) return -1;
  if (row_stride % 8 || row_stride < (Hq + Hk) * dk + Hk * dv || (v_first && first_stride % 8)) return -1;
  if (rot < 0 || rot % 2 || rot > d || (rot > 0 && (!rope || table_rows <= 0)) || page_size <= 0) return -1;
  int L = 1;
  while (L * 8 < max(dk, dv)) L *= 2;
  QkvFinishParams p{T_, Hq, Hk, d, dk, dv, rot, row_stride, page_size, L, table_rows, eps, lambda, first_stride, q_norm, k_norm,
                    reinterpret_cast<const float2*>(rope), positions, slots};
  const int heads = Hq + 2 * Hk, per_warp = 32 / L;
  const long long warps = (long long)(T_) * ((heads + per_warp - 1) / per_warp);
  MFQ_BY_TYPE(fp32, launch_kernel(qkv_finish_kernel<T>, dim3(unsigned((warps + 7) / 8)), dim3(256), 0, stream, static_cast<const T*>(qkv),
                                  static_cast<const T*>(v_first), static_cast<T*>(q_out), static_cast<T*>(k_pages),
                                  static_cast<T*>(v_pages), p));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// fp32 residual stream of a decoder (sublayers normalised on their input or on their output), and the per-head stage between
// the q/k/v projection and attention, for activations in bf16 or fp32.
//
//   embed_scaled      x = table[id] * scale              -> fp32 stream + copy in the activation type
//   norm_add          x += rms_norm(y) * w               -> fp32 stream + copy in the activation type, one pass over y and x
//   norm_out          h = rms_norm(x) * w                -> activation type (input of a sublayer or of the LM head)
//   qkv_finish        per head: RMS norm of q and k, rotation of the leading channels, blending of v with the values another
//                     layer computed for the same token, or RMS norm and rotation of v, K / V into their pages
//   turn_back         rotation of attention outputs by minus their position (for values that were rotated by theirs)
//   map_difference    differential attention: rms_norm(a1 - lambda a2) * scale of every head
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
// qkv rows [Hq * dk | Hk * maps * dk | Hk * dv] (dk, dv: head widths as stored, multiples of 16; d: the true q / k width the
// norm averages over; Hq counts every query map).  `L` lanes (a power of two) share a head, 8 channels each; a warp takes 32 / L
// heads of one token.  Queries may also be multiplied by a temperature that grows with the position.  The rotation reads (cos, sin) of the token's position from a table [positions][rot / 2]; channel i turns
// with i + rot / 2 (read from shared memory), or with its neighbour (`pairs`).  With v_d > 0 values are divided by their root mean
// square over v_d channels and all of these are rotated, from a table of their own.  Pages: K [page][Hk][16][maps * dk],
// V [page][Hk][16][dv]; slot < 0: the token is not cached.  No pages: rows hold queries only.
// ---------------------------------------------------------------------------------------------
struct QkvFinishParams {
  int T, Hq, Hk, maps, d, dk, dv, rot, pairs, row_stride, page_size, L, table_rows;
  float eps, lambda;        // lambda: share of the other layer's values
  float temp;               // queries times 1 + temp * ln(floor((position + 1) / temp_every) + 1)
  int temp_every;
  int first_stride;         // row stride of `v_first`
  const float* q_norm;
  const float* k_norm;      // [dk] fp32 or null: no norm
  const float2* rope;       // (cos, sin)
  const float2* v_rope;
  int v_d, v_table_rows;    // v_d 0: values stay as they are
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
  const int keys = k_pages ? p.Hk * p.maps : 0, heads = p.Hq + keys + (k_pages ? p.Hk : 0);
  const int groups = (heads + per_warp - 1) / per_warp;  // head groups of a token
  const int gw = blockIdx.x * 8 + warp;
  if (gw >= p.T * groups) return;  // whole warps leave together
  const int t = gw / groups, h = (gw - t * groups) * per_warp + sub;
  const bool live_head = h < heads;
  const bool is_q = h < p.Hq, is_v = h >= p.Hq + keys;
  const int width = is_v ? p.dv : p.dk;
  const bool mine = live_head && c * 8 < width;
  const T* row = qkv + size_t(t) * p.row_stride;
  const int col = is_v ? (p.Hq + keys) * p.dk + (h - p.Hq - keys) * p.dv : h * p.dk;
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
  if (is_v && p.v_d > 0) {
    const float inv = rsqrtf(ss / float(p.v_d) + p.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= inv;
  }
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
  const int rot = is_v ? p.v_d : p.rot;
  if (c * 8 < rot) {
    const int half = rot >> 1, pos = min(p.positions[t], (is_v ? p.v_table_rows : p.table_rows) - 1);
    const float2* tab = (is_v ? p.v_rope : p.rope) + size_t(pos) * half;
    if (p.pairs) {
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (c * 8 + j < rot) {
          const float2 cs = tab[(c * 8 + j) >> 1];
          const float a = v[j], b = v[j + 1];
          v[j] = a * cs.x - b * cs.y;
          v[j + 1] = b * cs.x + a * cs.y;
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (p.pairs) break;
      const int i = c * 8 + j;
      if (i < half) {
        const float2 cs = tab[i];
        v[j] = v[j] * cs.x - mysh[i + half] * cs.y;
      } else if (i < rot) {
        const float2 cs = tab[i - half];
        v[j] = v[j] * cs.x + mysh[i - half] * cs.y;
      }
    }
  }
  if (is_q) {
    if (p.temp != 0.f) {
      const float f = fmaf(p.temp, logf(float((p.positions[t] + 1) / p.temp_every) + 1.f), 1.f);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] *= f;
    }
    store8<T>(q_out + (size_t(t) * p.Hq + h) * p.dk + c * 8, v);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const int page = slot / p.page_size, off = slot - page * p.page_size;
  if (!is_v) {
    const int g = (h - p.Hq) / p.maps, m = h - p.Hq - g * p.maps;
    store8<T>(k_pages + (((size_t(page) * p.Hk + g) * p.page_size + off) * p.maps + m) * p.dk + c * 8, v);
    return;
  }
  const int g = h - p.Hq - keys;
  if (v_first) {
    float f[8];
    load8<T>(v_first + size_t(t) * p.first_stride + g * p.dv + c * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = (1.f - p.lambda) * v[j] + p.lambda * f[j];
  }
  store8<T>(v_pages + ((size_t(page) * p.Hk + g) * p.page_size + off) * p.dv + c * 8, v);
}

// ---------------------------------------------------------------------------------------------
// a [T][G][2][per][dv] (both maps of every head) -> out [T][G * per][dv]: y = a1 - lambda a2, out = scale * y / sqrt(mean(y^2) + eps),
// the mean over the `d` real channels (the others are zeros).  A warp per (token, head).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
map_difference_kernel(const T* __restrict__ a, T* __restrict__ out, int pairs, int H, int per, int dv, float inv_d, float lambda,
                      float scale, float eps) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (pair >= pairs) return;
  const int t = pair / H, h = pair - t * H, g = h / per, j = h - g * per;
  const bool mine = lane * 8 < dv;
  float y[8] = {};
  if (mine) {
    const T* a1 = a + ((size_t(t) * H + g * per) * 2 + j) * dv + lane * 8;
    float b[8];
    load8<T>(a1, y);
    load8<T>(a1 + size_t(per) * dv, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] -= lambda * b[i];
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += y[i] * y[i];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!mine) return;
  const float f = rsqrtf(ss * inv_d + eps) * scale;
#pragma unroll
  for (int i = 0; i < 8; ++i) y[i] *= f;
  store8<T>(out + size_t(pair) * dv + lane * 8, y);
}

// o [T][H][dv] in place: the pairs of the first 2 * half channels turn by minus the angle the table gives for the token's position.
// A thread takes kVec pairs (i, i + half) of a head, or kVec / 2 pairs of neighbours (`pairs`).
template <typename T, int kVec>
__global__ void __launch_bounds__(256)
turn_back_kernel(T* __restrict__ o, const float2* __restrict__ rope, const int* __restrict__ positions, int T_, int H, int dv, int half,
                 int table_rows, int pairs) {
  pdl_trigger();
  pdl_wait();
  const int per = (pairs ? 2 * half : half + kVec - 1) / kVec, items = H * per;
  const long long i = (long long)(blockIdx.x) * 256 + threadIdx.x;
  if (i >= (long long)(T_) * items) return;
  const int t = int(i / items), r = int(i - (long long)(t) * items), h = r / per, c = (r - h * per) * kVec;
  const float2* tab = rope + size_t(min(positions[t], table_rows - 1)) * half;
  T* head = o + (size_t(t) * H + h) * dv;
  if constexpr (kVec == 8) {
    float a[8], b[8];
    load8<T>(head + c, a);
    if (pairs) {
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        const float2 cs = tab[(c + j) >> 1];
        const float u = a[j], v = a[j + 1];
        a[j] = fmaf(u, cs.x, v * cs.y);
        a[j + 1] = fmaf(v, cs.x, -u * cs.y);
      }
    } else {
      load8<T>(head + c + half, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float2 cs = tab[c + j];
        const float u = a[j], v = b[j];
        a[j] = fmaf(u, cs.x, v * cs.y);
        b[j] = fmaf(v, cs.x, -u * cs.y);
      }
      store8<T>(head + c + half, b);
    }
    store8<T>(head + c, a);
  } else {
    const int lo = pairs ? c & ~1 : c, hi = pairs ? lo + 1 : c + half;
    if (pairs && (c & 1)) return;
    const float2 cs = tab[pairs ? lo >> 1 : lo];
    const float u = float(head[lo]), v = float(head[hi]);
    head[lo] = T(fmaf(u, cs.x, v * cs.y));
    head[hi] = T(fmaf(v, cs.x, -u * cs.y));
  }
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

extern "C" int mfq_map_difference(const void* a, void* out, int T_, int H, int per, int dv, int d, float lambda, float scale, float eps,
                                  int fp32, cudaStream_t stream) {
  if (T_ <= 0 || H <= 0 || per <= 0 || H % per || dv % 8 || dv <= 0 || dv > 256 || d <= 0 || d > dv) return -1;
  const long long pairs = (long long)(T_) * H;
  if (pairs > 0x7fffffff) return -1;
  MFQ_BY_TYPE(fp32, launch_kernel(map_difference_kernel<T>, dim3(unsigned((pairs + 7) / 8)), dim3(256), 0, stream,
                                  static_cast<const T*>(a), static_cast<T*>(out), int(pairs), H, per, dv, 1.f / float(d), lambda, scale, eps));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// o [T, H, dv] in place; rope [table_rows][d / 2] (cos, sin), d <= dv
extern "C" int mfq_turn_back(void* o, const float* rope, const int* positions, int T_, int H, int dv, int d, int table_rows, int pairs,
                             int fp32, cudaStream_t stream) {
  if (T_ <= 0 || H <= 0 || dv <= 0 || dv % 8 || d <= 0 || d % 2 || d > dv || !rope || table_rows <= 0) return -1;
  const int half = d / 2;
  const bool wide = pairs ? d % 8 == 0 : half % 8 == 0;
  const long long items = (long long)(T_) * H * (wide ? (pairs ? d / 8 : half / 8) : (pairs ? d : half));
  if ((items + 255) / 256 > 0x7fffffffLL) return -1;
  const float2* tab = reinterpret_cast<const float2*>(rope);
  const dim3 grid(unsigned((items + 255) / 256));
  if (wide)
    MFQ_BY_TYPE(fp32, launch_kernel(turn_back_kernel<T, 8>, grid, dim3(256), 0, stream, static_cast<T*>(o), tab, positions, T_, H, dv, half, table_rows, pairs));
  else
    MFQ_BY_TYPE(fp32, launch_kernel(turn_back_kernel<T, 1>, grid, dim3(256), 0, stream, static_cast<T*>(o), tab, positions, T_, H, dv, half, table_rows, pairs));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// k_pages null: the rows hold the Hq query heads only (Hk, dv unused).  v_d > 0: values are normed and rotated (v_rope [v_table_rows][v_d / 2])
extern "C" int mfq_qkv_finish(const void* qkv, int row_stride, const void* v_first, int first_stride, float lambda, void* q_out,
                              void* k_pages, void* v_pages, const int* positions, const int* slots, const float* q_norm,
                              const float* k_norm, const float* rope, int table_rows, int T_, int Hq, int Hk, int maps, int d, int dk,
                              int dv, int rot, int pairs, int page_size, float eps, float temp, int temp_every, const float* v_rope,
                              int v_d, int v_table_rows, int fp32, cudaStream_t stream) {
  if (temp != 0.f && temp_every <= 0) return -1;
  if (v_d < 0 || v_d % 2 || (v_d && (!k_pages || v_d > dv || !v_rope || v_table_rows <= 0 || v_first))) return -1;
  if (!k_pages) { Hk = 0; dv = 0; v_first = nullptr; }
  if (T_ <= 0 || Hq <= 0 || maps <= 0 || dk % 16 || dk <= 0 || dk > 256 || d <= 0 || d > dk) return -1;
  if (k_pages && (Hk <= 0 || Hq % (Hk * maps) || dv % 16 || dv <= 0 || dv > 256 || page_size <= 0 || !v_pages || !slots)) return -1;
  if (row_stride % 8 || row_stride < (Hq + Hk * maps) * dk + Hk * dv || (v_first && first_stride % 8)) return -1;
  if (rot < 0 || rot % 2 || rot > d || (rot > 0 && (!rope || table_rows <= 0))) return -1;
  int L = 1;
  while (L * 8 < max(dk, dv)) L *= 2;
  QkvFinishParams p{T_, Hq, Hk, maps, d, dk, dv, rot, pairs, row_stride, page_size, L, table_rows, eps, lambda, temp, temp_every, first_stride, q_norm, k_norm,
                    reinterpret_cast<const float2*>(rope), reinterpret_cast<const float2*>(v_rope), v_d, v_table_rows, positions, slots};
  const int heads = Hq + Hk * (maps + 1), per_warp = 32 / L;
  const long long warps = (long long)(T_) * ((heads + per_warp - 1) / per_warp);
  MFQ_BY_TYPE(fp32, launch_kernel(qkv_finish_kernel<T>, dim3(unsigned((warps + 7) / 8)), dim3(256), 0, stream, static_cast<const T*>(qkv),
                                  static_cast<const T*>(v_first), static_cast<T*>(q_out), static_cast<T*>(k_pages),
                                  static_cast<T*>(v_pages), p));
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// State-space recurrence token by token (see ssd.cuh for the equations): decode steps, short portions, and everything in fp32; and the
// gate and norm behind it.
//
//   ssd_recurrent_kernel   a CTA per (head, share of its columns, sequence) walks the tokens of the sequence's portion with the state in
//                          registers: a thread owns four adjacent columns on every R-th row.
//   ssd_gate_norm_kernel   a CTA per token: y silu(z), divided by its root mean square in equal runs of channels that may cross heads,
//                          times a weight
#include "ssd.cuh"

namespace mfq {

constexpr int kSsdThreads = 256;

// MAXR: rows a thread owns at most; CTAS per SM: many for a grid of several waves, few where the latency of one CTA counts
template <typename T, int MAXR, int CTAS>
__global__ void __launch_bounds__(kSsdThreads, CTAS)
ssd_recurrent_kernel(const T* __restrict__ x, const T* __restrict__ z, T* __restrict__ y, const SsdShape p, int split, int R) {
  pdl_trigger();
  extern __shared__ __align__(16) float ssd_sm[];
  const int N = p.N, P = p.P, H = p.H, cols = P / split, tid = threadIdx.x;
  const int h = blockIdx.x / split, c_base = blockIdx.x % split * cols, b = blockIdx.y, grp = h / (H / p.groups);
  float* b_s = ssd_sm;              // two stages of B [N], C [N], x [cols]
  const int stage = 2 * N + cols;
  float* part = ssd_sm + 2 * stage; // [R][cols]
  const int groups = cols / 4, cg = tid % groups, rg = tid / groups;
  const bool worker = rg < R;
  const float bias = p.dt_bias[h], rate = p.rate[h] * 1.4426950408889634f, skip = p.skip[h];
  pdl_wait();
  const int slot = p.slot[b];
  if (slot < 0) return;
  const int t0 = p.starts ? p.starts[b] : b, t1 = p.starts ? p.starts[b + 1] : b + 1;
  if (t0 >= t1) return;
  float* st = p.state + (size_t(slot) * H + h) * N * P + c_base + cg * 4;
  const int mine = worker ? (N - rg + R - 1) / R : 0;  // my rows: rg + R i
  float4 s[MAXR];
#pragma unroll
  for (int i = 0; i < MAXR; ++i)
    if (i < mine) s[i] = *reinterpret_cast<const float4*>(st + size_t(rg + R * i) * P);
  auto fetch = [&](int t) {
    const T* row = x + size_t(t) * p.x_stride;
    float* d = b_s + (t & 1) * stage;
    const T* bc = row + H * P + grp * N;
    for (int i = tid; i < N; i += kSsdThreads) {
      d[i] = to_float(bc[i]);
      d[N + i] = to_float(bc[p.groups * N + i]);
    }
    for (int i = tid; i < cols; i += kSsdThreads) d[2 * N + i] = to_float(row[h * P + c_base + i]);
  };
  fetch(t0);
  for (int t = t0; t < t1; ++t) {
    const float dt = ssd_softplus(to_float(z[size_t(t) * p.z_stride + h]) + bias), keep = exp2f(-rate * dt);
    __syncthreads();  // the token's vectors are there; everyone is done with the partial sums of the one before
    const float* d = b_s + (t & 1) * stage;
    if (t + 1 < t1) fetch(t + 1);
    if (worker) {
      float4 v = *reinterpret_cast<const float4*>(d + 2 * N + cg * 4), o = make_float4(0.f, 0.f, 0.f, 0.f);
      v.x *= dt; v.y *= dt; v.z *= dt; v.w *= dt;
#pragma unroll
      for (int i = 0; i < MAXR; ++i) {
        if (i < mine) {
          const float kb = d[rg + R * i], qc = d[N + rg + R * i];
          s[i].x = fmaf(keep, s[i].x, kb * v.x); s[i].y = fmaf(keep, s[i].y, kb * v.y);
          s[i].z = fmaf(keep, s[i].z, kb * v.z); s[i].w = fmaf(keep, s[i].w, kb * v.w);
          o.x = fmaf(qc, s[i].x, o.x); o.y = fmaf(qc, s[i].y, o.y);
          o.z = fmaf(qc, s[i].z, o.z); o.w = fmaf(qc, s[i].w, o.w);
        }
      }
      *reinterpret_cast<float4*>(part + rg * cols + cg * 4) = o;
    }
    __syncthreads();
    for (int c = tid; c < cols; c += kSsdThreads) {
      float o = skip * d[2 * N + c];
      for (int r = 0; r < R; ++r) o += part[r * cols + c];
      y[(size_t(t) * H + h) * P + c_base + c] = from_float<T>(o);
    }
  }
#pragma unroll
  for (int i = 0; i < MAXR; ++i)
    if (i < mine) *reinterpret_cast<float4*>(st + size_t(rg + R * i) * P) = s[i];
}

template <typename T, int MAXR, int CTAS>
static int launch_ssd_recurrent(const void* x, const void* z, void* y, const SsdShape& p, int B, int split, int R, cudaStream_t stream) {
  const int smem = (2 * (2 * p.N + p.P / split) + R * (p.P / split)) * 4;
  if (smem > 200 * 1024) return -5;
  static int allowed = 48 * 1024;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(ssd_recurrent_kernel<T, MAXR, CTAS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  launch_kernel(ssd_recurrent_kernel<T, MAXR, CTAS>, dim3(p.H * split, B), dim3(kSsdThreads), smem, stream, static_cast<const T*>(x), static_cast<const T*>(z),
                static_cast<T*>(y), p, split, R);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// y [T, H P], z (rows of z_stride) and w [H P] as stored; channel c of the true H * d lies at (c / d) P + c % d.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_gate_norm_kernel(const T* __restrict__ y, const T* __restrict__ z, const float* __restrict__ w, T* __restrict__ out, int H, int P, int d,
                     int z_stride, int parts, float eps) {
  pdl_trigger();
  extern __shared__ __align__(16) float gn_sm[];
  const int width = H * P, inner = H * d, per = inner / parts;
  float* v_s = gn_sm;             // [width]
  float* f_s = v_s + width;       // [parts]
  float* sum_s = f_s + parts;     // [max(parts, 8)]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t t = blockIdx.x;
  pdl_wait();
  for (int c = threadIdx.x * 8; c < width; c += 2048) {
    float a[8], g[8];
    load8<T>(y + t * width + c, a);
    load8<T>(z + t * z_stride + c, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] *= g[j] / (1.f + expf(-g[j]));
    store8<float>(v_s + c, a);
  }
  __syncthreads();
  const int each = max(1, 8 / parts);  // warps per part
  for (int j = warp; j < parts * each; j += 8) {
    const int part = j / each, n0 = part * per;
    float ss = 0.f;
    for (int i = (j - part * each) * 32 + lane; i < per; i += each * 32) {
      const int c = n0 + i;
      const float v = v_s[d == P ? c : c / d * P + c % d];
      ss = fmaf(v, v, ss);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) sum_s[j] = ss;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < parts; i += 256) {
    float ss = 0.f;
    for (int e = 0; e < each; ++e) ss += sum_s[i * each + e];
    f_s[i] = rsqrtf(ss / float(per) + eps);
  }
  __syncthreads();
  for (int c = threadIdx.x * 8; c < width; c += 2048) {
    float a[8], ww[8];
    load8<float>(v_s + c, a);
    load8<float>(w + c, ww);  // zero in padding channels
    const int head = c / P, n = head * d + c - head * P;  // 8 channels of a head; beyond the real ones w is zero
    if (per % 8 == 0 && d % 8 == 0) {
      const float f = f_s[min(n / per, parts - 1)];
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= f * ww[j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] *= f_s[min((n + j) / per, parts - 1)] * ww[j];
    }
    store8<T>(out + t * width + c, a);
  }
}

// The same where every part and head is a whole number of 8-channel vectors: a thread keeps its vectors in registers, and only their
// sums of squares go through shared memory.
template <typename T, int VECS>
__global__ void __launch_bounds__(512)
ssd_gate_norm_vec_kernel(const T* __restrict__ y, const T* __restrict__ z, const float* __restrict__ w, T* __restrict__ out, int H, int P, int d,
                         int z_stride, int parts, float eps) {
  pdl_trigger();
  extern __shared__ __align__(16) float gn_sm[];
  const int width = H * P, per = H * d / parts / 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  float* sum_s = gn_sm;              // [H d / 8] sums of squares of the real vectors
  float* f_s = sum_s + H * d / 8;    // [parts]
  const size_t t = blockIdx.x;
  int place[VECS];                   // of my vectors among the real ones; < 0: padding or none
  float ww[VECS][8];
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8, head = c / P, j = c - head * P;
    place[k] = c < width && j < d ? (head * d + j) / 8 : -1;
    if (c < width) load8<float>(w + c, ww[k]);
  }
  pdl_wait();
  float a[VECS][8];
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (place[k] >= 0) {
      float g[8], ss = 0.f;
      load8<T>(y + t * width + c, a[k]);
      load8<T>(z + t * z_stride + c, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        a[k][j] *= sizeof(T) == 4 ? g[j] / (1.f + expf(-g[j])) : __fdividef(g[j], 1.f + __expf(-fmaxf(g[j], -80.f)));
        ss = fmaf(a[k][j], a[k][j], ss);
      }
      sum_s[place[k]] = ss;
    }
  }
  __syncthreads();
  for (int i = warp; i < parts; i += warps) {
    float ss = 0.f;
    for (int j = lane; j < per; j += 32) ss += sum_s[i * per + j];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) f_s[i] = rsqrtf(ss / float(per * 8) + eps);
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < VECS; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c < width) {
      const float f = place[k] >= 0 ? f_s[place[k] / per] : 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) a[k][j] = place[k] >= 0 ? a[k][j] * f * ww[k][j] : 0.f;
      store8<T>(out + t * width + c, a[k]);
    }
  }
}

template <typename T>
static int launch_ssd_gate_norm(const void* y, const void* z, const float* w, void* out, int T_, int H, int P, int d, int z_stride, int parts, float eps,
                                cudaStream_t stream) {
  const int vecs = H * P / 8;
  if (d % 8 == 0 && H * d / parts % 8 == 0 && vecs <= 2048) {
    const int k = vecs <= 256 ? 1 : vecs <= 512 ? 2 : 4, threads = ((vecs + k - 1) / k + 31) / 32 * 32, bytes = (H * d / 8 + parts) * 4;
    auto run = [&](auto kernel) {
      launch_kernel(kernel, dim3(T_), dim3(threads), bytes, stream, static_cast<const T*>(y), static_cast<const T*>(z), w, static_cast<T*>(out), H, P, d,
                    z_stride, parts, eps);
    };
    if (k == 1) run(ssd_gate_norm_vec_kernel<T, 1>);
    else if (k == 2) run(ssd_gate_norm_vec_kernel<T, 2>);
    else run(ssd_gate_norm_vec_kernel<T, 4>);
    return cudaGetLastError() == cudaSuccess ? 0 : -7;
  }
  const int smem = (H * P + parts + max(parts, 8)) * 4;
  if (smem > 200 * 1024) return -5;
  static int allowed = 48 * 1024;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(ssd_gate_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  launch_kernel(ssd_gate_norm_kernel<T>, dim3(T_), dim3(256), smem, stream, static_cast<const T*>(y), static_cast<const T*>(z), w, static_cast<T*>(out),
                H, P, d, z_stride, parts, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace mfq

using namespace mfq;

// x [T, x_stride] as in ssd.cuh; z [T, z_stride]: dt before its bias in the first H columns; y [T, H P]; state fp32 [slots, H, N, P].
// starts null: one token per sequence.  split: CTAs over a head's columns.
extern "C" int mfq_ssd_recurrent(const void* x, const void* z, const float* dt_bias, const float* rate, const float* skip, void* y, float* state,
                                 const int* slot, const int* starts, int B, int H, int groups, int N, int P, int x_stride, int z_stride, int split,
                                 int fp32, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || H <= 0 || groups <= 0 || H % groups || N <= 0 || P <= 0 || N % 16 || P % 16) return -1;
  if (x_stride < H * P + 2 * groups * N || z_stride < H || split < 1 || P % (4 * split) || P / split / 4 > kSsdThreads) return -1;
  const int R = min(N, kSsdThreads / (P / split / 4)), rows = (N + R - 1) / R;
  if (rows > 16) return -5;
  const SsdShape p{H, groups, N, P, x_stride, z_stride, dt_bias, rate, skip, starts, slot, state};
  if (fp32) return launch_ssd_recurrent<float, 16, 1>(x, z, y, p, B, split, R, stream);
  if (rows > 8) return launch_ssd_recurrent<__nv_bfloat16, 16, 2>(x, z, y, p, B, split, R, stream);
  return H * split * B <= 4 * 148 ? launch_ssd_recurrent<__nv_bfloat16, 8, 2>(x, z, y, p, B, split, R, stream)
                                  : launch_ssd_recurrent<__nv_bfloat16, 8, 4>(x, z, y, p, B, split, R, stream);
}

// y [T, H P], z [T, z_stride], w [H P] fp32 (zero in padding channels), d of the P channels of a head are real; parts divides H * d.
extern "C" int mfq_ssd_gate_norm(const void* y, const void* z, const float* w, void* out, int T_, int H, int P, int d, int z_stride, int parts, float eps,
                                 int fp32, cudaStream_t stream) {
  if (T_ <= 0 || H <= 0 || P <= 0 || P % 16 || d <= 0 || d > P || z_stride % 8 || z_stride < H * P || parts <= 0 || (H * d) % parts) return -1;
  return fp32 ? launch_ssd_gate_norm<float>(y, z, w, out, T_, H, P, d, z_stride, parts, eps, stream)
              : launch_ssd_gate_norm<__nv_bfloat16>(y, z, w, out, T_, H, P, d, z_stride, parts, eps, stream);
}

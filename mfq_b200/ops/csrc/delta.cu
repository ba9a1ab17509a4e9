// Delta rule with a decay per key channel, token by token (see delta.cuh for the equations): decode steps, short portions, and
// everything in fp32.
//
//   delta_recurrent_kernel   a CTA per (head, sequence) walks the tokens of the sequence's portion with the state in registers (a
//                            thread owns four adjacent columns on every R-th row, at most 16 rows).  Unit norms, decays, write
//                            strength, norm and gate are fused in.  S^T k and S^T q are summed in one pass: o follows from the
//                            decayed state as S^T q + u (k . q).  The low-rank factors of a head's decays and gates are brought to
//                            shared memory ahead of the dependent-launch wait, if they fit.  The columns of a head may be split over a thread-block cluster,
//                            which adds its squares for the norm through distributed shared memory.
#include "delta.cuh"

namespace mfq {
namespace {

constexpr int kDeltaThreads = 256, kDeltaRows = 16, kDeltaMaxSplit = 8;

struct DeltaRecurrentParams {
  DeltaShape s;
  const int* starts;  // [B + 1] first token of every portion; null: token b is the portion of sequence b
  const int* slot;    // [B] state slot; < 0: skipped
  float* state;       // [slots, H, dk, dv]
  const float* dt_bias;  // [H dk]
  const float* rate;     // [H] exp(A_log)
  const float* norm_w;   // [dv]
  int split, rows;    // column split (cluster size); row groups R
  int staged;         // whether the factors lie in shared memory
};

__device__ __forceinline__ void delta_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
// n rows of `width` elements (a multiple of 8) to rows 16 bytes further apart
template <typename T>
__device__ __forceinline__ void delta_stage(T* dst, const T* src, int n, int width) {
  constexpr int kVec = 16 / sizeof(T);
  const int per = width / kVec;
  for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
    const int r = i / per, c = (i - r * per) * kVec;
    delta_cp16(dst + r * (width + kVec) + c, src + size_t(r) * width + c);
  }
}

__device__ __forceinline__ void delta_cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float delta_peer_load(const float* mine, uint32_t cta) {
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_u32(mine)), "r"(cta));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}
template <typename T>
__device__ __forceinline__ float delta_row_dot(const T* w, const float* x, int n, float z) {
  for (int r = 0; r < n; r += 8) {
    float v[8];
    load8<T>(w + r, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) z = fmaf(v[j], x[r + j], z);
  }
  return z;
}

template <typename T>
__global__ void __launch_bounds__(kDeltaThreads, 2)
delta_recurrent_kernel(const T* __restrict__ conv, const T* __restrict__ side, const T* __restrict__ w_a2, const T* __restrict__ w_g2,
                       T* __restrict__ y, const DeltaRecurrentParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) float dl_sm[];
  const int dk = p.s.dk, dv = p.s.dv, H = p.s.H;
  const int cols = dv / p.split, c_base = blockIdx.x % p.split * cols;
  const int h = blockIdx.x / p.split, b = blockIdx.y, kh = h / (H / p.s.G);
  const int R = p.rows;
  float* q_s = dl_sm;              // [dk]
  float* k_s = q_s + dk;           // [dk]
  float* d_s = k_s + dk;           // [dk] decay
  float* a_s = d_s + dk;           // [ra]
  float* g_s = a_s + p.s.ra;       // [rg]
  float* v_s = g_s + p.s.rg;       // [cols] value, then u / |k|
  float* gate_s = v_s + cols;      // [cols]
  float* part_k = gate_s + cols;   // [R][cols]
  float* part_q = part_k + R * cols;
  constexpr int kPad = 16 / sizeof(T);
  const T *a2 = w_a2 + size_t(h) * dk * p.s.ra, *g2 = w_g2 + (size_t(h) * dv + c_base) * p.s.rg;
  int a2_pitch = p.s.ra, g2_pitch = p.s.rg;
  if (p.staged) {
    T* sa = reinterpret_cast<T*>(part_q + R * cols);
    T* sg = sa + dk * (p.s.ra + kPad);
    delta_stage<T>(sa, a2, dk, p.s.ra);
    delta_stage<T>(sg, g2, cols, p.s.rg);
    a2 = sa; g2 = sg;
    a2_pitch += kPad; g2_pitch += kPad;
  }
  __shared__ float red[33];
  __shared__ float dots[8][3];
  __shared__ float ss_own[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int groups = cols / 4, cg = tid % groups, rg = tid / groups;
  const int mine = rg < R ? (dk - rg + R - 1) / R : 0;  // my rows: rg + R i
  pdl_wait();
  const int slot = p.slot[b];
  if (slot < 0) {  // the whole cluster leaves
    asm volatile("cp.async.wait_all;" ::: "memory");
    return;
  }
  const int t0 = p.starts ? p.starts[b] : b, t1 = p.starts ? p.starts[b + 1] : b + 1;
  float* st = p.state + (size_t(slot) * H + h) * dk * dv + c_base + cg * 4;
  float4 s[kDeltaRows];
#pragma unroll
  for (int i = 0; i < kDeltaRows; ++i)
    if (i < mine) s[i] = *reinterpret_cast<const float4*>(st + size_t(rg + R * i) * dv);
  const float rate = -1.4426950408889634f * p.rate[h];
  for (int t = t0; t < t1; ++t) {
    const T* row = conv + size_t(t) * p.s.conv_stride;
    const T* srow = side + size_t(t) * p.s.side_stride;
    for (int i = tid; i < p.s.ra + p.s.rg; i += kDeltaThreads) a_s[i] = to_float(srow[p.s.b_cols + i]);  // a, then g
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int i = tid; i < dk; i += kDeltaThreads) {
      const float q = to_float(row[kh * dk + i]), k = to_float(row[(p.s.G + kh) * dk + i]);
      q_s[i] = q;
      k_s[i] = k;
      qq = fmaf(q, q, qq);
      kk = fmaf(k, k, kk);
      qk = fmaf(q, k, qk);
    }
    for (int i = tid; i < cols; i += kDeltaThreads) v_s[i] = to_float(row[2 * p.s.G * dk + h * dv + c_base + i]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
      qk += __shfl_xor_sync(0xffffffffu, qk, o);
    }
    if (lane == 0) { dots[warp][0] = qq; dots[warp][1] = kk; dots[warp][2] = qk; }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    qq = kk = qk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { qq += dots[w][0]; kk += dots[w][1]; qk += dots[w][2]; }
    const float iq = rsqrtf(qq + 1e-6f) * p.s.scale, ik = rsqrtf(kk + 1e-6f), beta = delta_sigmoid(to_float(srow[h]));
    for (int i = tid; i < dk + cols; i += kDeltaThreads) {  // decays of the rows, then gates of my columns
      if (i < dk) {
        const float z = delta_row_dot<T>(a2 + i * a2_pitch, a_s, p.s.ra, p.dt_bias[h * dk + i]);
        d_s[i] = exp2f(fmaxf(rate * delta_softplus(z), kGlaFloor));
      } else {
        gate_s[i - dk] = delta_sigmoid(delta_row_dot<T>(g2 + (i - dk) * g2_pitch, g_s, p.s.rg, 0.f));
      }
    }
    __syncthreads();
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
    for (int i = 0; i < kDeltaRows; ++i) {
      if (i < mine) {
        const int r = rg + R * i;
        const float d = d_s[r], k = k_s[r], q = q_s[r];
        s[i].x *= d; s[i].y *= d; s[i].z *= d; s[i].w *= d;
        ak.x = fmaf(k, s[i].x, ak.x); ak.y = fmaf(k, s[i].y, ak.y); ak.z = fmaf(k, s[i].z, ak.z); ak.w = fmaf(k, s[i].w, ak.w);
        aq.x = fmaf(q, s[i].x, aq.x); aq.y = fmaf(q, s[i].y, aq.y); aq.z = fmaf(q, s[i].z, aq.z); aq.w = fmaf(q, s[i].w, aq.w);
      }
    }
    if (rg < R) {
      *reinterpret_cast<float4*>(part_k + rg * cols + cg * 4) = ak;
      *reinterpret_cast<float4*>(part_q + rg * cols + cg * 4) = aq;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < cols; c += kDeltaThreads) {
      float sk = 0.f, sq = 0.f;
      for (int r = 0; r < R; ++r) { sk += part_k[r * cols + c]; sq += part_q[r * cols + c]; }
      const float u = beta * (v_s[c] - ik * sk), o = iq * fmaf(u * ik, qk, sq);
      v_s[c] = u * ik;
      part_q[c] = o;  // row 0 of this column is read by this thread only
      ss += o * o;
    }
    ss = dense_block_sum(ss, red);
    {
      const float4 u = rg < R ? *reinterpret_cast<const float4*>(v_s + cg * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < kDeltaRows; ++i) {
        if (i < mine) {
          const float k = k_s[rg + R * i];
          s[i].x = fmaf(k, u.x, s[i].x); s[i].y = fmaf(k, u.y, s[i].y); s[i].z = fmaf(k, u.z, s[i].z); s[i].w = fmaf(k, u.w, s[i].w);
        }
      }
    }
    if (p.split > 1) {
      if (tid == 0) ss_own[t & 1] = ss;
      delta_cluster_barrier();
      ss = 0.f;
      for (int z = 0; z < p.split; ++z) ss += delta_peer_load(&ss_own[t & 1], z);
    }
    const float f = rsqrtf(ss * p.s.inv_dv + p.s.eps);
    for (int c = tid; c < cols; c += kDeltaThreads)
      y[(size_t(t) * H + h) * dv + c_base + c] = from_float<T>(part_q[c] * f * p.norm_w[c_base + c] * gate_s[c]);
    __syncthreads();  // the token's vectors are replaced next
  }
#pragma unroll
  for (int i = 0; i < kDeltaRows; ++i)
    if (i < mine) *reinterpret_cast<float4*>(st + size_t(rg + R * i) * dv) = s[i];
  if (p.split > 1) delta_cluster_barrier();  // nobody leaves while a peer still reads its sum
}

template <typename T>
int launch_delta_recurrent(const void* conv, const void* side, const void* w_a2, const void* w_g2, void* y, const DeltaRecurrentParams& p0, int B,
                           cudaStream_t stream) {
  const int cols = p0.s.dv / p0.split, pad = 16 / int(sizeof(T));
  const int plain = (3 * p0.s.dk + p0.s.ra + p0.s.rg + 2 * cols + 2 * p0.rows * cols) * 4;
  const int factors = (p0.s.dk * (p0.s.ra + pad) + cols * (p0.s.rg + pad)) * int(sizeof(T));
  DeltaRecurrentParams p = p0;
  p.staged = plain + factors <= 100 * 1024;  // two CTAs per SM
  const int smem = plain + (p.staged ? factors : 0);
  if (smem > 200 * 1024) return -5;
  static int allowed = 48 * 1024;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(delta_recurrent_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  const dim3 grid(p.s.H * p.split, B), block(kDeltaThreads);
  const T *c = static_cast<const T*>(conv), *sd = static_cast<const T*>(side), *wa = static_cast<const T*>(w_a2), *wg = static_cast<const T*>(w_g2);
  const cudaError_t rc = p.split > 1
      ? launch_kernel_clustered(delta_recurrent_kernel<T>, grid, block, dim3(p.split), smem, stream, c, sd, wa, wg, static_cast<T*>(y), p)
      : launch_kernel(delta_recurrent_kernel<T>, grid, block, smem, stream, c, sd, wa, wg, static_cast<T*>(y), p);
  return rc == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace
}  // namespace mfq

using namespace mfq;

// conv [T, conv_stride], side [T, side_stride] as in delta.cuh; w_a2 [H dk, ra], w_g2 [H dv, rg] in the element type; dt_bias [H dk],
// rate [H], norm_w [dv] fp32; y [T, H dv]; state fp32 [slots, H, dk, dv].  starts null: one token per sequence.  split: cluster size
// over a head's columns; a thread holds at most 16 state rows.
extern "C" int mfq_delta_recurrent(const void* conv, const void* side, const void* w_a2, const void* w_g2, const float* dt_bias,
                                   const float* rate, const float* norm_w, void* y, float* state, const int* slot, const int* starts, int B,
                                   int H, int G, int dk, int dv, int real_dv, int b_cols, int ra, int rg, int conv_stride, int side_stride,
                                   int split, float scale, float eps, int fp32, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || dk % 16 || dv % 16 || real_dv <= 0 || real_dv > dv) return -1;
  if (b_cols < H || b_cols % 8 || ra <= 0 || rg <= 0 || ra % 8 || rg % 8 || conv_stride < 2 * G * dk + H * dv || side_stride < b_cols + ra + rg) return -1;
  if (split < 1 || split > kDeltaMaxSplit || dv % (4 * split)) return -1;
  const int groups = dv / split / 4;
  if (groups > kDeltaThreads) return -1;
  const int rows = min(dk, kDeltaThreads / groups);
  if ((dk + rows - 1) / rows > kDeltaRows) return -5;
  const DeltaRecurrentParams p{DeltaShape{H, G, dk, dv, b_cols, ra, rg, conv_stride, side_stride, scale, 1.f / float(real_dv), eps}, starts, slot,
                               state, dt_bias, rate, norm_w, split, rows, 0};
  return fp32 ? launch_delta_recurrent<float>(conv, side, w_a2, w_g2, y, p, B, stream)
              : launch_delta_recurrent<__nv_bfloat16>(conv, side, w_a2, w_g2, y, p, B, stream);
}

// Gated linear attention, token by token (see gla.cuh for the equations): decode steps, short portions, and everything in fp32.
//
//   gla_recurrent_kernel   a CTA per (head, sequence) walks the tokens of the sequence's portion.  A thread owns four adjacent
//                          state columns on every R-th row; the state streams through registers (read and written once per
//                          token), the first rows are requested before the token's decays are evaluated.  Decays, norm and
//                          gate are fused in.  With few (head, sequence) pairs the columns of a head are split over a thread
//                          block cluster, which adds its squares for the norm through distributed shared memory.
#include "gla.cuh"

namespace mfq {

constexpr int kGlaThreads = 256, kGlaAhead = 8, kGlaMaxSplit = 8;

struct GlaRecurrentParams {
  GlaShape s;
  const int* starts;  // [B + 1] first token of every portion; null: token b is the portion of sequence b
  const int* slot;    // [B] state slot; < 0: skipped
  float* state;       // [slots, H, dk, dv]
  int split, rows;    // column split (cluster size); row groups R
};

__device__ __forceinline__ void gla_cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float gla_peer_load(const float* mine, uint32_t cta) {
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_u32(mine)), "r"(cta));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}

template <typename T>
__global__ void __launch_bounds__(kGlaThreads)
gla_recurrent_kernel(const T* __restrict__ proj, const T* __restrict__ w2, const float* __restrict__ bias,
                     const float* __restrict__ norm_w, T* __restrict__ y, const GlaRecurrentParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) float gla_sm[];
  const int dk = p.s.dk, dv = p.s.dv, rank = p.s.rank, H = p.s.H;
  const int cols = dv / p.split, c_base = blockIdx.x % p.split * cols;  // my state columns
  const int h = blockIdx.x / p.split, b = blockIdx.y;
  float* q_s = gla_sm;           // [dk]
  float* k_s = q_s + dk;         // [dk]
  float* d_s = k_s + dk;         // [dk] decay
  float* u_s = d_s + dk;         // [dk] bonus
  float* a_s = u_s + dk;         // [rank]
  float* v_s = a_s + rank;       // [cols]
  float* part = v_s + cols;      // [R][cols]
  __shared__ float red[33];
  __shared__ float ss_own[2];
  const int tid = threadIdx.x;
  const int groups = cols / 4, R = p.rows;
  const int cg = tid % groups, rg = tid / groups;
  const bool worker = rg < R;
  pdl_wait();
  const int slot = p.slot[b];
  if (slot < 0) return;  // the whole cluster leaves
  const int t0 = p.starts ? p.starts[b] : b, t1 = p.starts ? p.starts[b + 1] : b + 1;
  float* st = p.state + (size_t(slot) * H + h) * dk * dv + c_base + cg * 4;
  const int mine = worker ? (dk - rg + R - 1) / R : 0;  // my rows: rg + R i
  for (int t = t0; t < t1; ++t) {
    const T* row = proj + size_t(t) * p.s.row_stride;
    float4 s[kGlaAhead];
#pragma unroll
    for (int i = 0; i < kGlaAhead; ++i)
      if (i < mine) s[i] = *reinterpret_cast<const float4*>(st + size_t(rg + R * i) * dv);
    for (int i = tid; i < rank; i += kGlaThreads) a_s[i] = to_float(row[2 * H * (dk + dv) + i]);
    for (int i = tid; i < dk; i += kGlaThreads) {
      q_s[i] = to_float(row[h * dk + i]) * p.s.scale;
      k_s[i] = to_float(row[(H + h) * dk + i]);
    }
    for (int i = tid; i < cols; i += kGlaThreads) v_s[i] = to_float(row[2 * H * dk + h * dv + c_base + i]);
    __syncthreads();
    for (int i = tid; i < dk; i += kGlaThreads) {
      const T* w = w2 + size_t(h * dk + i) * rank;
      float z = bias[h * dk + i];
      for (int r = 0; r < rank; r += 8) {
        float x[8];
        load8<T>(w + r, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) z = fmaf(x[j], a_s[r + j], z);
      }
      d_s[i] = exp2f(gla_log2_decay(p.s, z));
      if (p.s.bonus) u_s[i] = p.s.bonus[h * dk + i];
    }
    __syncthreads();
    if (worker) {
      const float4 v = *reinterpret_cast<const float4*>(v_s + cg * 4);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int i0 = 0; i0 < mine; i0 += kGlaAhead) {
        if (i0 > 0) {
#pragma unroll
          for (int i = 0; i < kGlaAhead; ++i)
            if (i0 + i < mine) s[i] = *reinterpret_cast<const float4*>(st + size_t(rg + R * (i0 + i)) * dv);
        }
#pragma unroll
        for (int i = 0; i < kGlaAhead; ++i) {
          if (i0 + i < mine) {
            const int r = rg + R * (i0 + i);
            const float q = q_s[r], k = k_s[r], d = d_s[r];
            if (p.s.bonus) {  // read-out before the write
              const float uk = u_s[r] * k;
              o.x = fmaf(q, fmaf(uk, v.x, s[i].x), o.x); o.y = fmaf(q, fmaf(uk, v.y, s[i].y), o.y);
              o.z = fmaf(q, fmaf(uk, v.z, s[i].z), o.z); o.w = fmaf(q, fmaf(uk, v.w, s[i].w), o.w);
            }
            s[i].x = fmaf(d, s[i].x, k * v.x); s[i].y = fmaf(d, s[i].y, k * v.y);
            s[i].z = fmaf(d, s[i].z, k * v.z); s[i].w = fmaf(d, s[i].w, k * v.w);
            if (!p.s.bonus) {
              o.x = fmaf(q, s[i].x, o.x); o.y = fmaf(q, s[i].y, o.y);
              o.z = fmaf(q, s[i].z, o.z); o.w = fmaf(q, s[i].w, o.w);
            }
            *reinterpret_cast<float4*>(st + size_t(r) * dv) = s[i];
          }
        }
      }
      *reinterpret_cast<float4*>(part + rg * cols + cg * 4) = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < cols; c += kGlaThreads) {
      float o = 0.f;
      for (int r = 0; r < R; ++r) o += part[r * cols + c];
      part[c] = o;  // row 0 of this column is read by this thread only
      ss += o * o;
    }
    ss = dense_block_sum(ss, red);
    if (p.split > 1) {
      if (tid == 0) ss_own[t & 1] = ss;
      gla_cluster_barrier();
      ss = 0.f;
      for (int z = 0; z < p.split; ++z) ss += gla_peer_load(&ss_own[t & 1], z);
    }
    const float f = rsqrtf(ss * p.s.inv_dv + p.s.eps);
    for (int c = tid; c < cols; c += kGlaThreads) {
      const float gate = to_float(row[2 * H * dk + (H + h) * dv + c_base + c]);
      y[(size_t(t) * H + h) * dv + c_base + c] = from_float<T>(part[c] * f * norm_w[h * p.s.norm_stride + c_base + c] * silu_of(gate));
    }
    __syncthreads();  // the token's vectors are replaced next
  }
  if (p.split > 1) gla_cluster_barrier();  // nobody leaves while a peer still reads its sum
}

template <typename T>
static int launch_gla_recurrent(const void* proj, const void* w2, const float* bias, const float* norm_w, void* y,
                                const GlaRecurrentParams& p, int B, cudaStream_t stream) {
  const int smem = (4 * p.s.dk + p.s.rank + (1 + p.rows) * (p.s.dv / p.split)) * 4;
  if (smem > 200 * 1024) return -5;
  static int allowed = 48 * 1024;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(gla_recurrent_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  const dim3 grid(p.s.H * p.split, B), block(kGlaThreads);
  const cudaError_t rc = p.split > 1
      ? launch_kernel_clustered(gla_recurrent_kernel<T>, grid, block, dim3(p.split), smem, stream, static_cast<const T*>(proj),
                                static_cast<const T*>(w2), bias, norm_w, static_cast<T*>(y), p)
      : launch_kernel(gla_recurrent_kernel<T>, grid, block, smem, stream, static_cast<const T*>(proj), static_cast<const T*>(w2), bias,
                      norm_w, static_cast<T*>(y), p);
  return rc == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace mfq

using namespace mfq;

// proj [T, row_stride] as in gla.cuh; w2 [H * dk, rank]; bias and bonus (may be null) [H * dk] and norm_w [dv] (norm_stride 0) or
// [H, dv] fp32; y [T, H * dv]; state fp32
// [slots, H, dk, dv].  starts null: one token per sequence.  split: cluster size over a head's columns.
extern "C" int mfq_gla_recurrent(const void* proj, const void* w2, const float* bias, const float* norm_w, void* y, float* state,
                                 const int* slot, const int* starts, int B, int H, int dk, int dv, int real_dv, int rank,
                                 int row_stride, int split, float scale, float inv_tau, float eps, int decay, int norm_stride,
                                 const float* bonus, int fp32, cudaStream_t stream) {
  if (decay < kGlaSigmoid || decay > kGlaExp || (norm_stride && norm_stride != dv)) return -1;
  if (B <= 0 || B > 65535 || H <= 0 || dk <= 0 || dv <= 0 || dk % 16 || dv % 16 || rank <= 0 || rank % 8 || real_dv <= 0 || real_dv > dv) return -1;
  if (row_stride < 2 * H * (dk + dv) + rank || row_stride % 8 || split < 1 || split > kGlaMaxSplit || dv % (4 * split)) return -1;
  const int groups = dv / split / 4;
  if (groups > kGlaThreads) return -1;
  GlaRecurrentParams p{GlaShape{H, dk, dv, rank, row_stride, scale, inv_tau, 1.f / float(real_dv), eps, decay, norm_stride, bonus}, starts, slot, state, split,
                       min(dk, kGlaThreads / groups)};
  return fp32 ? launch_gla_recurrent<float>(proj, w2, bias, norm_w, y, p, B, stream)
              : launch_gla_recurrent<__nv_bfloat16>(proj, w2, bias, norm_w, y, p, B, stream);
}

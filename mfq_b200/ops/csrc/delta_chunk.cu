// Delta rule with a decay per key channel over prompt portions in 64-token chunks, bf16 (see delta.cuh for the recurrence).
//
// With b_t the running sum of g inside a chunk, S_0 the state before it, C its length, and K, Q, V the chunk's rows,
//   (I + L) U = beta V - (beta 2^b K) S_0,        L_ts = beta_t sum_c k_tc k_sc 2^(b_tc - b_sc)   (s < t)
//   =>  U = U_0 - W S_0,   U_0 = (I + L)^-1 beta V,   W = (I + L)^-1 (beta 2^b K)
//   O   = (2^b Q) S_0 + P U,                      P_ts = sum_c q_tc k_sc 2^(b_tc - b_sc)          (s <= t)
//   S_C = diag(2^b_C) S_0 + (2^(b_C - b) K)^T U
// which is the token recurrence unrolled over the chunk.  Three kernels:
//
//   delta_chunk_prepare   a CTA per (chunk, head), every chunk in parallel: unit norms, decays and their running sum b, L and P, the
//                         unit-triangular system by forward substitution with a column of [beta V | beta 2^b K] per thread (64
//                         registers, fp32), and the operand tiles of the scan
//   delta_chunk_scan      the only sequential part: a CTA per (head, 32 state columns) walks the chunks with the fp32 state slice in
//                         accumulator registers; per chunk W S_0, Q S_0, P U and K^T U.  A tile lies in global memory as in shared
//                         memory, so it arrives by one cp.async.bulk copy on an mbarrier.  Waits are bounded.
//   delta_norm_gate       per-head norm and gate of the raw outputs
//
// Scores (L, P) are formed in 16 x 16 blocks relative to b before the block's first row, where both factors are at most 1 below the
// diagonal; a diagonal block whose own decay spans more than 2^-100 is summed term by term instead.  Every fp32 operand of a product
// is split into two bf16 numbers (16 significant bits), so the recurrence keeps fp32-level sums; v, and q and k before their norms,
// are bf16 as they come.  The 16-row products are too small for 128-row tcgen05 tiles and the chain per chunk is latency-bound, so
// they run as mma.sync.
#include "chunk_ops.cuh"
#include "delta.cuh"

namespace mfq {
namespace {

constexpr int kDcThreads = 256, kDcWarps = 8, kDcMaxDk = 128, kDcMaxRank = 64;
constexpr int kDcPp = 72;   // row pitch of P (bf16)
constexpr int kDcLp = 68;   // row pitch of L (fp32)
constexpr int kDcNs = 32;   // state columns per CTA of the scan
constexpr int kDcBp = 40;   // row pitch of the state copy and of U in the scan (bf16)

struct DeltaChunkParams {
  DeltaShape s;
  const __nv_bfloat16* conv;   // [T, conv_stride]
  const __nv_bfloat16* side;   // [T, side_stride]
  const __nv_bfloat16* w_a2;   // [H dk, ra]
  const float* dt_bias;        // [H dk]
  const float* rate;           // [H]
  const int* starts;           // [B + 1] first token of every portion
  const int* slot;             // [B]
  float* state;                // [slots, H, dk, dv]
  __nv_bfloat16* wq;           // [chunks, H] tiles: W hi, W lo, Q hi, Q lo, each [64][dk + 8]
  __nv_bfloat16* kp;           // [chunks, H] tiles: K hi, K lo [64][dk + 8], P hi, P lo [64][72], 2^b_C [dk] fp32
  float* u0;                   // [chunks, H, 64, dv]
  float* o_raw;                // [T, H dv]
  int* status;
};

// Elements (bf16) of the tiles.
__host__ __device__ constexpr int dc_wq(int dk) { return 4 * kGc * (dk + 8); }
__host__ __device__ constexpr int dc_kp(int dk) { return 2 * kGc * (dk + 8) + 2 * kGc * kDcPp + 2 * dk; }

struct DeltaChunkAt {
  int t0, n;
  size_t index;
};
__device__ __forceinline__ bool dc_locate(const DeltaChunkParams& p, int chunk, int b, DeltaChunkAt& at) {
  const int r0 = p.starts[b], len = p.starts[b + 1] - r0;
  at.t0 = r0 + chunk * kGc;
  at.n = min(kGc, len - chunk * kGc);
  at.index = size_t((r0 - p.starts[0]) / kGc + b + chunk);
  return at.n > 0 && p.slot[b] >= 0;
}
__device__ __forceinline__ float dc_softplus(float z) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + gc_exp2(-1.4426950408889634f * fabsf(z))));
  return fmaf(0.6931471805599453f, y, fmaxf(z, 0.f));
}

struct DeltaPrepareSmem {
  int b, q, k, l, misc, bytes;
};
__host__ __device__ inline DeltaPrepareSmem dc_prepare_smem(int dk) {
  DeltaPrepareSmem m{};
  m.b = 0;                                   // [64][dk + 8] fp32
  m.q = m.b + kGc * (dk + 8) * 4;            // q, k [64][dk + 8] bf16
  m.k = m.q + kGc * (dk + 8) * 2;
  m.l = m.k + kGc * (dk + 8) * 2;            // a [64][rank + 8] bf16, then L [64][68] fp32
  m.misc = m.l + kGc * kDcLp * 4;            // iq, ik, beta [64], totals [256] fp32
  m.bytes = m.misc + (3 * kGc + kDcThreads) * 4;
  return m;
}

__global__ void __launch_bounds__(kDcThreads, 2)
delta_chunk_prepare_kernel(const DeltaChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t dc_sm[];
  pdl_wait();
  DeltaChunkAt at;
  if (!dc_locate(p, blockIdx.x, blockIdx.z, at)) return;
  const int h = blockIdx.y, H = p.s.H, G = p.s.G, dk = p.s.dk, dv = p.s.dv, rank = p.s.ra, kh = h / (H / G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const DeltaPrepareSmem m = dc_prepare_smem(dk);
  float* b_s = reinterpret_cast<float*>(dc_sm + m.b);
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.q);
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.k);
  __nv_bfloat16* a_s = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.l);
  float* l_s = reinterpret_cast<float*>(dc_sm + m.l);
  float* iq_s = reinterpret_cast<float*>(dc_sm + m.misc);
  float *ik_s = iq_s + kGc, *beta_s = ik_s + kGc, *tot = beta_s + kGc;
  const int bp = dk + 8, kp = dk + 8;
  const __nv_bfloat16* rows = p.conv + size_t(at.t0) * p.s.conv_stride;
  const __nv_bfloat16* side = p.side + size_t(at.t0) * p.s.side_stride;
  gc_rows<kDcWarps>(a_s, rank + 8, side + p.s.b_cols, p.s.side_stride, rank, at.n, warp, lane);
  gc_commit();
  gc_rows<kDcWarps>(q_s, kp, rows + kh * dk, p.s.conv_stride, dk, at.n, warp, lane);
  gc_rows<kDcWarps>(k_s, kp, rows + (G + kh) * dk, p.s.conv_stride, dk, at.n, warp, lane);
  gc_commit();
  if (tid < kGc) beta_s[tid] = tid < at.n ? delta_sigmoid(__bfloat162float(side[size_t(tid) * p.s.side_stride + h])) : 0.f;
  gc_wait<1>();
  __syncthreads();
  // ----- decays, then their running sum: a thread takes one key channel of 64 / TG tokens -----
  {
    const float rate = -1.4426950408889634f * p.rate[h];
    const float* dt = p.dt_bias + h * dk;
    gc_low_rank<kDcWarps>(a_s, rank + 8, p.w_a2 + size_t(h) * dk * rank, rank, dk, warp, lane, [&](int t, int c, float x, float y) {
      const float2 bias = *reinterpret_cast<const float2*>(dt + c);
      const bool in = t < at.n;
      *reinterpret_cast<float2*>(b_s + t * bp + c) = make_float2(in ? fmaxf(rate * dc_softplus(x + bias.x), kGlaFloor) : 0.f,
                                                                 in ? fmaxf(rate * dc_softplus(y + bias.y), kGlaFloor) : 0.f);
    });
  }
  __syncthreads();
  const int TG = dk <= 32 ? 8 : dk <= 64 ? 4 : 2, len = kGc / TG, c = tid % dk, tg = tid / dk;
  const bool live = tg < TG;
  if (live) {
    float run = 0.f;
#pragma unroll 8
    for (int t = tg * len; t < tg * len + len; ++t) {
      run += b_s[t * bp + c];
      b_s[t * bp + c] = run;
    }
    tot[tg * dk + c] = run;
  }
  gc_wait<0>();
  __syncthreads();
  __nv_bfloat16* tile_kp = p.kp + (at.index * H + h) * size_t(dc_kp(dk));
  __nv_bfloat16* tile_wq = p.wq + (at.index * H + h) * size_t(dc_wq(dk));
  if (live && tg > 0) {
    float off = 0.f;
    for (int i = 0; i < tg; ++i) off += tot[i * dk + c];
    for (int t = tg * len; t < tg * len + len; ++t) b_s[t * bp + c] += off;
  }
  for (int t = warp; t < kGc; t += kDcWarps) {
    float qq = 0.f, kk = 0.f;
    for (int i = lane * 2; i < dk; i += 64) {
      const float2 q = gc_pair(q_s + t * kp + i), k = gc_pair(k_s + t * kp + i);
      qq = fmaf(q.x, q.x, fmaf(q.y, q.y, qq));
      kk = fmaf(k.x, k.x, fmaf(k.y, k.y, kk));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
    }
    if (lane == 0) {
      iq_s[t] = rsqrtf(qq + 1e-6f) * p.s.scale;
      ik_s[t] = rsqrtf(kk + 1e-6f);
    }
  }
  __syncthreads();
  // ----- L and P: warp = row block I and one half of the column blocks J <= I; the second half is taken in reverse -----
  __nv_bfloat16 *p_hi = tile_kp + 2 * kGc * kp, *p_lo = p_hi + kGc * kDcPp;
  bool wide = false;
  {
    const bool upper = warp & 4;
    const int I = upper ? 3 - (warp & 3) : warp & 3, J0 = upper ? (I + 2) / 2 : 0, J1 = upper ? I + 1 : (I + 2) / 2;  // J0 .. J1 - 1
    float aq[2][2][4] = {}, ak[2][2][4] = {};
    const float* ref = b_s + (16 * I - 1) * bp;
    for (int ks = 0; ks < dk / 16 && J0 < J1; ++ks) {
      uint32_t qh[4], ql[4], kh_[4], kl_[4];
      float2 rf[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int cc = ks * 16 + e * 8 + t4 * 2;
        rf[e] = I ? *reinterpret_cast<const float2*>(ref + cc) : make_float2(0.f, 0.f);
        const float2 last = *reinterpret_cast<const float2*>(b_s + (16 * I + 15) * bp + cc);
        wide = wide || rf[e].x - last.x > kGcSpan || rf[e].y - last.y > kGcSpan;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = 16 * I + r * 8 + g;
          const float2 q = gc_pair(q_s + t * kp + cc), k = gc_pair(k_s + t * kp + cc), b = *reinterpret_cast<const float2*>(b_s + t * bp + cc);
          const float ex = gc_exp2(b.x - rf[e].x), ey = gc_exp2(b.y - rf[e].y);
          gc_split(q.x * ex, q.y * ey, qh[e * 2 + r], ql[e * 2 + r]);
          gc_split(k.x * ex, k.y * ey, kh_[e * 2 + r], kl_[e * 2 + r]);
        }
      }
#pragma unroll
      for (int jj = 0; jj < 2; ++jj) {
        if (J0 + jj < J1) {
          uint32_t sh[2][2], sl[2][2];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int s = 16 * (J0 + jj) + nt * 8 + g;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int cc = ks * 16 + e * 8 + t4 * 2;
              const float2 k = gc_pair(k_s + s * kp + cc), b = *reinterpret_cast<const float2*>(b_s + s * bp + cc);
              gc_split(k.x * gc_exp2(rf[e].x - b.x), k.y * gc_exp2(rf[e].y - b.y), sh[nt][e], sl[nt][e]);
            }
          }
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) { gc_mma(aq[jj][nt], qh, sh[nt][0], sh[nt][1]); gc_mma(ak[jj][nt], kh_, sh[nt][0], sh[nt][1]); }
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) { gc_mma(aq[jj][nt], ql, sh[nt][0], sh[nt][1]); gc_mma(ak[jj][nt], kl_, sh[nt][0], sh[nt][1]); }
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) { gc_mma(aq[jj][nt], qh, sl[nt][0], sl[nt][1]); gc_mma(ak[jj][nt], kh_, sl[nt][0], sl[nt][1]); }
        }
      }
    }
    // (the last reader of a is behind a barrier: L may take its place)
#pragma unroll
    for (int jj = 0; jj < 2; ++jj)
      if (J0 + jj < J1)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int t = 16 * I + r * 8 + g, s = 16 * (J0 + jj) + nt * 8 + t4 * 2;
            const float ft = beta_s[t] * ik_s[t], fq = iq_s[t], s0 = ik_s[s], s1 = ik_s[s + 1];
            *reinterpret_cast<float2*>(l_s + t * kDcLp + s) =
                make_float2(s < t ? ft * s0 * ak[jj][nt][2 * r] : 0.f, s + 1 < t ? ft * s1 * ak[jj][nt][2 * r + 1] : 0.f);
            const float x = s <= t ? fq * s0 * aq[jj][nt][2 * r] : 0.f, y = s + 1 <= t ? fq * s1 * aq[jj][nt][2 * r + 1] : 0.f;
            gc_split(x, y, *reinterpret_cast<uint32_t*>(p_hi + t * kDcPp + s), *reinterpret_cast<uint32_t*>(p_lo + t * kDcPp + s));
          }
  }
  if (__syncthreads_or(wide)) {  // diagonal blocks term by term
    for (int i = tid; i < 4 * 256; i += kDcThreads) {
      const int t = (i >> 8) * 16 + ((i >> 4) & 15), s = (i >> 8) * 16 + (i & 15);
      if (s > t) continue;
      float xq = 0.f, xk = 0.f;
      for (int cc = 0; cc < dk; ++cc) {
        const float ks = __bfloat162float(k_s[s * kp + cc]) * gc_exp2(b_s[t * bp + cc] - b_s[s * bp + cc]);
        xq = fmaf(__bfloat162float(q_s[t * kp + cc]), ks, xq);
        xk = fmaf(__bfloat162float(k_s[t * kp + cc]), ks, xk);
      }
      xq *= iq_s[t] * ik_s[s];
      l_s[t * kDcLp + s] = s < t ? beta_s[t] * ik_s[t] * ik_s[s] * xk : 0.f;
      const __nv_bfloat16 hi = __float2bfloat16(xq);
      p_hi[t * kDcPp + s] = hi;
      p_lo[t * kDcPp + s] = __float2bfloat16(xq - __bfloat162float(hi));
    }
    __syncthreads();
  }
  // ----- Q and K of the scan, 2^b_C -----
  {
    __nv_bfloat16 *q_hi = tile_wq + 2 * kGc * kp, *q_lo = q_hi + kGc * kp, *k_hi = tile_kp, *k_lo = k_hi + kGc * kp;
    float* gam = reinterpret_cast<float*>(tile_kp + 2 * kGc * kp + 2 * kGc * kDcPp);
    for (int i = tid; i < dk; i += kDcThreads) gam[i] = gc_exp2(b_s[(kGc - 1) * bp + i]);
    for (int t = warp; t < kGc; t += kDcWarps) {
      const float fq = iq_s[t], fk = ik_s[t];
      for (int cc = lane * 2; cc < dk; cc += 64) {
        const float2 q = gc_pair(q_s + t * kp + cc), k = gc_pair(k_s + t * kp + cc), b = *reinterpret_cast<const float2*>(b_s + t * bp + cc);
        const float2 e = *reinterpret_cast<const float2*>(b_s + (kGc - 1) * bp + cc);
        gc_split(q.x * fq * gc_exp2(b.x), q.y * fq * gc_exp2(b.y), *reinterpret_cast<uint32_t*>(q_hi + t * kp + cc), *reinterpret_cast<uint32_t*>(q_lo + t * kp + cc));
        gc_split(k.x * fk * gc_exp2(e.x - b.x), k.y * fk * gc_exp2(e.y - b.y), *reinterpret_cast<uint32_t*>(k_hi + t * kp + cc),
                 *reinterpret_cast<uint32_t*>(k_lo + t * kp + cc));
      }
    }
  }
  // ----- (I + L) x = right-hand side, a column per thread: [beta V | beta 2^b K] -----
  float* u0 = p.u0 + (at.index * H + h) * size_t(kGc) * dv;
  __nv_bfloat16 *w_hi = tile_wq, *w_lo = w_hi + kGc * kp;
  const __nv_bfloat16* v = rows + 2 * G * dk + h * dv;
  for (int col = tid; col < dv + dk; col += kDcThreads) {
    float x[kGc];
    if (col < dv) {
#pragma unroll
      for (int i = 0; i < kGc; ++i) x[i] = i < at.n ? beta_s[i] * __bfloat162float(v[size_t(i) * p.s.conv_stride + col]) : 0.f;
    } else {
      const int cc = col - dv;
#pragma unroll
      for (int i = 0; i < kGc; ++i) x[i] = beta_s[i] * ik_s[i] * gc_exp2(b_s[i * bp + cc]) * __bfloat162float(k_s[i * kp + cc]);
    }
#pragma unroll
    for (int i = 1; i < kGc; ++i) {
      float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
      for (int j = 0; j + 3 < i; j += 4) {
        const float4 l4 = *reinterpret_cast<const float4*>(l_s + i * kDcLp + j);
        a0 = fmaf(l4.x, x[j], a0);
        a1 = fmaf(l4.y, x[j + 1], a1);
        a2 = fmaf(l4.z, x[j + 2], a2);
        a3 = fmaf(l4.w, x[j + 3], a3);
      }
#pragma unroll
      for (int j = i & ~3; j < i; ++j) a0 = fmaf(l_s[i * kDcLp + j], x[j], a0);
      x[i] -= (a0 + a1) + (a2 + a3);
    }
    if (col < dv) {
#pragma unroll
      for (int i = 0; i < kGc; ++i) u0[size_t(i) * dv + col] = x[i];
    } else {
      const int cc = col - dv;
#pragma unroll
      for (int i = 0; i < kGc; ++i) {
        const __nv_bfloat16 hi = __float2bfloat16(x[i]);
        w_hi[i * kp + cc] = hi;
        w_lo[i * kp + cc] = __float2bfloat16(x[i] - __bfloat162float(hi));
      }
    }
  }
}

struct DeltaScanSmem {
  int wq, kp, s, d, bars, bytes;
};
__host__ __device__ inline DeltaScanSmem dc_scan_smem(int dk) {
  DeltaScanSmem m{};
  m.wq = 0;
  m.kp = m.wq + dc_wq(dk) * 2;          // two buffers
  m.s = m.kp + 2 * dc_kp(dk) * 2;       // hi, lo [dk][40]
  m.d = m.s + 2 * dk * kDcBp * 2;       // hi, lo [64][40]
  m.bars = m.d + 2 * kGc * kDcBp * 2;
  m.bytes = m.bars + 64;
  return m;
}

__device__ __forceinline__ void dc_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(src)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

__global__ void __launch_bounds__(kDcThreads, 1)
delta_chunk_scan_kernel(const DeltaChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t dc_sm[];
  const int h = blockIdx.y, b = blockIdx.z, H = p.s.H, dk = p.s.dk, dv = p.s.dv, kp = dk + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mat = lane >> 3, mrow = lane & 7;
  const DeltaScanSmem m = dc_scan_smem(dk);
  __nv_bfloat16* wq_s = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.wq);
  __nv_bfloat16* kp_s = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.kp);
  __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.s);
  __nv_bfloat16* s_lo = s_hi + dk * kDcBp;
  __nv_bfloat16* d_hi = reinterpret_cast<__nv_bfloat16*>(dc_sm + m.d);
  __nv_bfloat16* d_lo = d_hi + kGc * kDcBp;
  uint64_t* bars = reinterpret_cast<uint64_t*>(dc_sm + m.bars);  // [0] W / Q, [1], [2] K / P buffers
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 3);
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  pdl_wait();
  const int slot = p.slot[b], r0 = p.starts[b], len = p.starts[b + 1] - r0;
  if (slot < 0 || len <= 0) return;
  const int chunks = (len + kGc - 1) / kGc, col0 = blockIdx.x * kDcNs, tiles = min(kDcNs, dv - col0) / 8;  // 2 or 4 column tiles
  const size_t first = size_t((r0 - p.starts[0]) / kGc + b);
  __syncthreads();
  const uint32_t wq_bytes = dc_wq(dk) * 2, kp_bytes = dc_kp(dk) * 2;
  auto load_wq = [&](int c) {
    mbar_expect_tx(&bars[0], wq_bytes);
    dc_bulk(wq_s, p.wq + ((first + c) * H + h) * size_t(dc_wq(dk)), wq_bytes, &bars[0]);
  };
  auto load_kp = [&](int c) {
    mbar_expect_tx(&bars[1 + (c & 1)], kp_bytes);
    dc_bulk(kp_s + (c & 1) * dc_kp(dk), p.kp + ((first + c) * H + h) * size_t(dc_kp(dk)), kp_bytes, &bars[1 + (c & 1)]);
  };
  if (tid == 0) {
    load_wq(0);
    load_kp(0);
    if (chunks > 1) load_kp(1);
  }
  // state slice: warp w owns rows 16 w + {g, g + 8}, all column tiles
  const bool has_rows = warp * 16 < dk;
  float* st = p.state + (size_t(slot) * H + h) * dk * dv + col0;
  float s[4][4] = {};
  auto publish = [&]() {
    if (!has_rows) return;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      const int off = (16 * warp + g) * kDcBp + 8 * nt + 2 * t4;
      gc_split(s[nt][0], s[nt][1], *reinterpret_cast<uint32_t*>(s_hi + off), *reinterpret_cast<uint32_t*>(s_lo + off));
      gc_split(s[nt][2], s[nt][3], *reinterpret_cast<uint32_t*>(s_hi + off + 8 * kDcBp), *reinterpret_cast<uint32_t*>(s_lo + off + 8 * kDcBp));
    }
  };
  if (has_rows) {
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      if (nt < tiles) {
        const float2 lo = *reinterpret_cast<const float2*>(st + size_t(16 * warp + g) * dv + 8 * nt + 2 * t4);
        const float2 hi = *reinterpret_cast<const float2*>(st + size_t(16 * warp + g + 8) * dv + 8 * nt + 2 * t4);
        s[nt][0] = lo.x; s[nt][1] = lo.y; s[nt][2] = hi.x; s[nt][3] = hi.y;
      }
    }
  }
  publish();
  __syncthreads();
  const int mt = warp >> 1, nt0 = 2 * (warp & 1);  // my token rows 16 mt + {g, g + 8} and my two column tiles
  const bool my_tiles = nt0 < tiles;
  const int i0 = 16 * mt + g, i1 = i0 + 8;
  const uint32_t frag = ((mt * 16 + (mat & 1) * 8 + mrow) * kp + (mat >> 1) * 8) * 2;          // A operand rows of W and Q
  const uint32_t pfrag = ((mt * 16 + (mat & 1) * 8 + mrow) * kDcPp + (mat >> 1) * 8) * 2;      // ... of P
  const uint32_t bfrag = (((mat & 1) * 8 + mrow) * kDcBp + (mat >> 1) * 8) * 2;                // B operand, two column tiles
  const uint32_t kfrag = (((mat >> 1) * 8 + mrow) * kp + 16 * warp + (mat & 1) * 8) * 2;       // A operand K^T of the update
  const uint32_t wa = smem_u32(wq_s), plane = uint32_t(kGc * kp) * 2, sa_hi = smem_u32(s_hi), sa_lo = smem_u32(s_lo), da_hi = smem_u32(d_hi),
                 da_lo = smem_u32(d_lo);
  bool ok = true;
  for (int c = 0; c < chunks; ++c) {
    const int t0 = r0 + c * kGc, n = min(kGc, len - c * kGc);
    const float* u0 = p.u0 + ((first + c) * H + h) * size_t(kGc) * dv + col0;
    float2 u[2][2];
#pragma unroll
    for (int nn = 0; nn < 2; ++nn) {
      u[nn][0] = my_tiles ? *reinterpret_cast<const float2*>(u0 + size_t(i0) * dv + 8 * (nt0 + nn) + 2 * t4) : make_float2(0.f, 0.f);
      u[nn][1] = my_tiles ? *reinterpret_cast<const float2*>(u0 + size_t(i1) * dv + 8 * (nt0 + nn) + 2 * t4) : make_float2(0.f, 0.f);
    }
    ok = mbar_wait(&bars[0], c & 1, abort_flag, p.status, kStatusTimeoutProducer) && ok;
    ok = mbar_wait(&bars[1 + (c & 1)], (c >> 1) & 1, abort_flag, p.status, kStatusTimeoutProducer) && ok;
    const __nv_bfloat16* kt = kp_s + (c & 1) * dc_kp(dk);
    const float* gam = reinterpret_cast<const float*>(kt + 2 * kGc * kp + 2 * kGc * kDcPp);
    // ----- W S and Q S -----
    float ws[2][4] = {}, o[2][4] = {};
    if (my_tiles) {
      for (int ks = 0; ks < dk / 16; ++ks) {
        uint32_t wh[4], wl[4], qh[4], ql[4], sh[4], sl[4];
        gc_ldm(wa + frag + ks * 32, wh);
        gc_ldm(wa + plane + frag + ks * 32, wl);
        gc_ldm(wa + 2 * plane + frag + ks * 32, qh);
        gc_ldm(wa + 3 * plane + frag + ks * 32, ql);
        const uint32_t off = bfrag + (ks * 16 * kDcBp + nt0 * 8) * 2;
        gc_ldm_t(sa_hi + off, sh);
        gc_ldm_t(sa_lo + off, sl);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) { gc_mma(ws[nn], wh, sh[2 * nn], sh[2 * nn + 1]); gc_mma(o[nn], qh, sh[2 * nn], sh[2 * nn + 1]); }
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) { gc_mma(ws[nn], wl, sh[2 * nn], sh[2 * nn + 1]); gc_mma(o[nn], ql, sh[2 * nn], sh[2 * nn + 1]); }
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) { gc_mma(ws[nn], wh, sl[2 * nn], sl[2 * nn + 1]); gc_mma(o[nn], qh, sl[2 * nn], sl[2 * nn + 1]); }
      }
    }
#pragma unroll
    for (int nn = 0; nn < 2; ++nn) {
      const int off = i0 * kDcBp + 8 * (nt0 + nn) + 2 * t4;
      gc_split(u[nn][0].x - ws[nn][0], u[nn][0].y - ws[nn][1], *reinterpret_cast<uint32_t*>(d_hi + off), *reinterpret_cast<uint32_t*>(d_lo + off));
      gc_split(u[nn][1].x - ws[nn][2], u[nn][1].y - ws[nn][3], *reinterpret_cast<uint32_t*>(d_hi + off + 8 * kDcBp),
               *reinterpret_cast<uint32_t*>(d_lo + off + 8 * kDcBp));
    }
    if (!__syncthreads_and(ok)) break;  // U visible; W, Q and the state copy are free
    if (tid == 0 && c + 1 < chunks) {
      fence_proxy_async_smem();
      load_wq(c + 1);
    }
    // ----- O += P U over the causal blocks, then the state -----
    const uint32_t pa = smem_u32(kt + 2 * kGc * kp), pplane = uint32_t(kGc * kDcPp) * 2, ka = smem_u32(kt);
    if (my_tiles) {
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t ph[4], pl[4], uh[4], ul[4];
        gc_ldm(pa + pfrag + ks * 32, ph);
        gc_ldm(pa + pplane + pfrag + ks * 32, pl);
        const uint32_t off = bfrag + (ks * 16 * kDcBp + nt0 * 8) * 2;
        gc_ldm_t(da_hi + off, uh);
        gc_ldm_t(da_lo + off, ul);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) gc_mma(o[nn], ph, uh[2 * nn], uh[2 * nn + 1]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) gc_mma(o[nn], pl, uh[2 * nn], uh[2 * nn + 1]);
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) gc_mma(o[nn], ph, ul[2 * nn], ul[2 * nn + 1]);
      }
      float* orow = p.o_raw + size_t(t0) * H * dv + h * dv + col0;
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
        const int cc = 8 * (nt0 + nn) + 2 * t4;
        if (i0 < n) *reinterpret_cast<float2*>(orow + size_t(i0) * H * dv + cc) = make_float2(o[nn][0], o[nn][1]);
        if (i1 < n) *reinterpret_cast<float2*>(orow + size_t(i1) * H * dv + cc) = make_float2(o[nn][2], o[nn][3]);
      }
    }
    if (has_rows) {
      const float g0 = gam[16 * warp + g], g1 = gam[16 * warp + g + 8];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) { s[nt][0] *= g0; s[nt][1] *= g0; s[nt][2] *= g1; s[nt][3] *= g1; }
#pragma unroll
      for (int ks = 0; ks < kGc / 16; ++ks) {
        uint32_t kh[4], kl[4], uh[2][4], ul[2][4];
        gc_ldm_t(ka + kfrag + ks * 16 * kp * 2, kh);
        gc_ldm_t(ka + plane + kfrag + ks * 16 * kp * 2, kl);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const uint32_t off = bfrag + (ks * 16 * kDcBp + i * 16) * 2;
          gc_ldm_t(da_hi + off, uh[i]);
          gc_ldm_t(da_lo + off, ul[i]);
        }
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) gc_mma(s[nt], kh, uh[nt >> 1][(nt & 1) * 2], uh[nt >> 1][(nt & 1) * 2 + 1]);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) gc_mma(s[nt], kl, uh[nt >> 1][(nt & 1) * 2], uh[nt >> 1][(nt & 1) * 2 + 1]);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) gc_mma(s[nt], kh, ul[nt >> 1][(nt & 1) * 2], ul[nt >> 1][(nt & 1) * 2 + 1]);
      }
      publish();
    }
    __syncthreads();  // the new state copy is visible; the K / P buffer and U are free
    if (tid == 0 && c + 2 < chunks) {
      fence_proxy_async_smem();
      load_kp(c + 2);
    }
  }
  if (!ok) {
    // a copy may still be in flight towards this CTA's shared memory: give it one more bounded wait
    if (tid == 0) {
      const unsigned long long w0 = globaltimer_ns();
      while (globaltimer_ns() - w0 < 2000000ull) {
      }
    }
    __syncthreads();
    return;  // the state is left as it was; the host sees the status word
  }
  if (has_rows) {
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      if (nt < tiles) {
        *reinterpret_cast<float2*>(st + size_t(16 * warp + g) * dv + 8 * nt + 2 * t4) = make_float2(s[nt][0], s[nt][1]);
        *reinterpret_cast<float2*>(st + size_t(16 * warp + g + 8) * dv + 8 * nt + 2 * t4) = make_float2(s[nt][2], s[nt][3]);
      }
    }
  }
}

// y = rms_norm(o) * w * sigmoid(gate); L lanes (a power of two) per (token, head)
__global__ void __launch_bounds__(256)
delta_norm_gate_kernel(const float* __restrict__ o, const __nv_bfloat16* __restrict__ gate, const float* __restrict__ norm_w,
                       __nv_bfloat16* __restrict__ y, int pairs, int dv, int L, float inv_dv, float eps) {
  pdl_trigger();
  pdl_wait();
  const int pair = (blockIdx.x * 256 + threadIdx.x) / L, lane = threadIdx.x & (L - 1);
  const bool live = pair < pairs;
  const size_t at = size_t(live ? pair : 0) * dv;
  constexpr int kMost = 4;  // 8-wide vectors per lane: values up to 1024 wide
  float v[kMost][8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < kMost; ++i) {
    const int c = (lane + i * L) * 8;
    if (c < dv) {
      load8<float>(o + at + c, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[i][j] * v[i][j];
    }
  }
  for (int i = L >> 1; i > 0; i >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, i);
  if (!live) return;
  const float f = rsqrtf(ss * inv_dv + eps);
#pragma unroll
  for (int i = 0; i < kMost; ++i) {
    const int c = (lane + i * L) * 8;
    if (c < dv) {
      float w[8], z[8];
      load8<__nv_bfloat16>(gate + at + c, z);
      load8<float>(norm_w + c, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= f * w[j] * __fdividef(1.f, 1.f + __expf(-fmaxf(z[j], -80.f)));
      store8<__nv_bfloat16>(y + at + c, v[i]);
    }
  }
}

}  // namespace
}  // namespace mfq

using namespace mfq;

// Bytes of scratch per (chunk, head); `chunks` of a call are T / 64 + B for portions of T tokens.
extern "C" long long mfq_delta_chunk_bytes(int dk, int dv) {
  return (dc_wq(dk) + dc_kp(dk)) * 2ll + 1ll * kGc * dv * 4;
}

// Portions of B sequences (tokens starts[b] .. starts[b + 1] - 1 of conv, side, gate and y), longest `max_q`; arguments as
// mfq_delta_recurrent.  gate [T, H dv]: the gate's logits of tokens first .. first + count - 1 are read; o_raw [T, H dv] fp32 and
// scratch (chunks * H * mfq_delta_chunk_bytes) are work space.  Returns -5 for sizes that do not fit.
extern "C" int mfq_delta_chunk(const void* conv, const void* side, const void* w_a2, const void* gate, const float* dt_bias, const float* rate,
                               const float* norm_w, void* y, float* state, const int* slot, const int* starts, float* o_raw, void* scratch,
                               int chunks, int first, int count, int B, int max_q, int H, int G, int dk, int dv, int real_dv, int b_cols, int ra,
                               int rg, int conv_stride, int side_stride, float scale, float eps, int* status, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || max_q <= 0 || H <= 0 || H > 65535 || G <= 0 || H % G || dk <= 0 || dv <= 0 || dk % 16 || dv % 16 || real_dv <= 0 || real_dv > dv) return -1;
  if (b_cols < H || b_cols % 8 || ra <= 0 || ra % 8 || conv_stride % 8 || side_stride % 8 || conv_stride < 2 * G * dk + H * dv || chunks <= 0 || count <= 0) return -1;
  const int prep = dc_prepare_smem(dk).bytes, scan = dc_scan_smem(dk).bytes;
  if (dk > kDcMaxDk || dv > 1024 || ra > kDcMaxRank || ra % 16 || scan > 227 * 1024) return -5;
  const size_t tiles = size_t(chunks) * H;
  __nv_bfloat16* wq = static_cast<__nv_bfloat16*>(scratch);
  __nv_bfloat16* kp = wq + tiles * dc_wq(dk);
  float* u0 = reinterpret_cast<float*>(kp + tiles * dc_kp(dk));
  const DeltaChunkParams p{DeltaShape{H, G, dk, dv, b_cols, ra, rg, conv_stride, side_stride, scale, 1.f / float(real_dv), eps},
                           static_cast<const __nv_bfloat16*>(conv), static_cast<const __nv_bfloat16*>(side), static_cast<const __nv_bfloat16*>(w_a2),
                           dt_bias, rate, starts, slot, state, wq, kp, u0, o_raw, status};
  static int allowed_prep = 0, allowed_scan = 0;
  if (prep > allowed_prep) {
    if (cudaFuncSetAttribute(delta_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, prep) != cudaSuccess) return -6;
    allowed_prep = prep;
  }
  if (scan > allowed_scan) {
    if (cudaFuncSetAttribute(delta_chunk_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, scan) != cudaSuccess) return -6;
    allowed_scan = scan;
  }
  launch_kernel(delta_chunk_prepare_kernel, dim3((max_q + kGc - 1) / kGc, H, B), dim3(kDcThreads), prep, stream, p);
  launch_kernel(delta_chunk_scan_kernel, dim3((dv + kDcNs - 1) / kDcNs, H, B), dim3(kDcThreads), scan, stream, p);
  const long long pairs = (long long)(count) * H;
  const size_t skip = size_t(first) * H * dv;
  int lanes = 1;
  while (lanes * 8 < dv && lanes < 32) lanes *= 2;
  launch_kernel(delta_norm_gate_kernel, dim3(unsigned((pairs * lanes + 255) / 256)), dim3(256), 0, stream, o_raw + skip, static_cast<const __nv_bfloat16*>(gate) + skip,
                norm_w, static_cast<__nv_bfloat16*>(y) + skip, int(pairs), dv, lanes, 1.f / float(real_dv), eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// Gated linear attention over prompt portions in 64-token chunks, bf16 (see gla.cuh for the recurrence).
//
// With b_t the running sum of g inside a chunk, S_0 the state before it and C its length,
//     o_t = (2^b_t q_t)^T S_0 + sum_{s <= t} A_ts v_s,       A_ts = sum_c q_tc k_sc 2^(b_tc - b_sc)
//     S_C = diag(2^b_C) S_0 + U,                             U    = sum_s (2^(b_C - b_s) k_s) v_s^T
// so all that is sequential is one multiply-add per state element and chunk.  Three kernels:
//
//   gla_chunk_local    a CTA per (chunk, head): decays and their running sum b, and U
//   gla_chunk_state    a thread per eight state elements: replaces every U by the S_0 of its chunk, advances the state
//   gla_chunk_output   a CTA per (chunk, head): A, then O = A V + (2^b q)^T S_0, per-head norm and gate
//
// With a bonus u the query of token t stands before its own write: b_(t-1) takes the place of b_t beside q, A is strictly lower
// triangular, and its diagonal is sum_c q_tc u_c k_tc.
//
// Exponents never overflow: A is formed in 16 x 16 blocks relative to b before the block's first row, where both factors are at
// most 1 below the diagonal; a diagonal block whose own decay spans more than 2^-100 is summed term by term instead.
// Precision: the recurrence is kept to fp32 level on bf16 tensor cores by splitting every fp32 operand into two bf16 numbers
// (16 significant bits): 2^(b_C - b) k, 2^b q, the factors of A, A itself and S_0; v is bf16 as projected.  The 16-row
// products here are too small for 128-row tcgen05 tiles, and their operands are made in registers, so they run as mma.sync.
#include "chunk_ops.cuh"
#include "gla.cuh"

#include <type_traits>

namespace mfq {
namespace {

constexpr int kGcThreads = 512, kGcWarps = kGcThreads / 32, kGcMaxDk = 256, kGcMaxDv = 512;

struct GlaChunkParams {
  GlaShape s;
  const __nv_bfloat16* proj;  // [T, row_stride]
  const __nv_bfloat16* w2;    // [H dk, rank]
  const float* bias;          // [H dk]
  const float* norm_w;        // [dv]
  __nv_bfloat16* y;           // [T, H dv]
  const int* starts;          // [B + 1] first token of every portion
  const int* slot;            // [B]
  float* state;               // [slots, H, dk, dv]
  float* cum;                 // [T, H dk]           b
  float* u;                   // [chunks, H, dk, dv] U, then S_0 as [hi x 8 | lo x 8] bf16 per eight elements
  float* gam;                 // [chunks, H, dk]     2^b_C
};

// log2(sigmoid(z)) and silu to a few units of 2^-23 (absolute, relative)
__device__ __forceinline__ float gc_log2_sigmoid(float z) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + gc_exp2(-1.4426950408889634f * fabsf(z))));
  return fmaf(1.4426950408889634f, fminf(z, 0.f), -y);
}
__device__ __forceinline__ float gc_log2_decay(const GlaShape& s, float z) {
  if (s.decay == kGlaSigmoid) return gc_log2_sigmoid(z) * s.inv_tau;
  return fmaxf(-1.4426950408889634f * gc_exp2(1.4426950408889634f * z), kGlaFloor);
}
__device__ __forceinline__ float gc_silu(float x) { return __fdividef(x, 1.f + gc_exp2(-1.4426950408889634f * fmaxf(x, -80.f))); }
// A CTA's chunk: tokens t0 .. t0 + n - 1; `index` numbers the chunks of all portions without overlap.
struct GlaChunkAt {
  int t0, n;
  size_t index;
};
__device__ __forceinline__ bool gc_locate(const GlaChunkParams& p, int chunk, int b, GlaChunkAt& at) {
  const int r0 = p.starts[b], len = p.starts[b + 1] - r0;
  at.t0 = r0 + chunk * kGc;
  at.n = min(kGc, len - chunk * kGc);
  at.index = size_t((r0 - p.starts[0]) / kGc + b + chunk);
  return at.n > 0 && p.slot[b] >= 0;
}

__host__ __device__ constexpr int gc_groups(int dk) { return dk <= 64 ? 8 : dk <= 128 ? 4 : 2; }

struct GlaLocalSmem {
  int b, k, lo, v, tot, bytes;
};
__host__ __device__ inline GlaLocalSmem gc_local_smem(int dk, int dv, int rank) {
  GlaLocalSmem m{};
  m.b = 0;                                                   // [64][dk + 8] fp32
  m.k = m.b + kGc * (dk + 8) * 4;                            // a [64][rank + 8] bf16, then hi [64][dk + 8] bf16
  const int half = kGc * (dk + 8) * 2, abytes = kGc * (rank + 8) * 2;
  m.lo = m.k + (half > abytes ? half : abytes);              // k, then lo [64][dk + 8] bf16
  m.v = m.lo + half;                                         // [64][dv + 8] bf16
  m.tot = m.v + kGc * (dv + 8) * 2;                          // [512] fp32
  m.bytes = m.tot + kGcThreads * 4;
  return m;
}

__global__ void __launch_bounds__(kGcThreads, 2)
gla_chunk_local_kernel(const GlaChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t gc_sm[];
  pdl_wait();
  GlaChunkAt at;
  if (!gc_locate(p, blockIdx.x, blockIdx.z, at)) return;
  const int h = blockIdx.y, H = p.s.H, dk = p.s.dk, dv = p.s.dv, rank = p.s.rank;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const GlaLocalSmem m = gc_local_smem(dk, dv, rank);
  float* b_s = reinterpret_cast<float*>(gc_sm + m.b);
  __nv_bfloat16* a_s = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.k);
  __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.k);
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.v);
  float* tot = reinterpret_cast<float*>(gc_sm + m.tot);
  const int bp = dk + 8, kp = dk + 8, vp = dv + 8;
  __nv_bfloat16* k_lo = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.lo);
  const __nv_bfloat16* rows = p.proj + size_t(at.t0) * p.s.row_stride;
  gc_rows<kGcWarps>(a_s, rank + 8, rows + 2 * H * (dk + dv), p.s.row_stride, rank, at.n, warp, lane);
  gc_commit();
  gc_rows<kGcWarps>(k_lo, kp, rows + (H + h) * dk, p.s.row_stride, dk, at.n, warp, lane);
  gc_commit();
  gc_rows<kGcWarps>(v_s, vp, rows + 2 * H * dk + h * dv, p.s.row_stride, dv, at.n, warp, lane);
  gc_commit();
  gc_wait<2>();
  __syncthreads();
  // ----- decays, then their running sum: a thread takes one key channel of 64 / TG tokens -----
  {
    const float* bias = p.bias + h * dk;
    gc_low_rank<kGcWarps>(a_s, rank + 8, p.w2 + size_t(h) * dk * rank, rank, dk, warp, lane, [&](int t, int c, float x, float y) {
      const float2 add = *reinterpret_cast<const float2*>(bias + c);
      const bool in = t < at.n;
      *reinterpret_cast<float2*>(b_s + t * bp + c) = make_float2(in ? gc_log2_decay(p.s, x + add.x) : 0.f, in ? gc_log2_decay(p.s, y + add.y) : 0.f);
    });
  }
  __syncthreads();
  const int TG = gc_groups(dk), len = kGc / TG, c = tid % dk, tg = tid / dk;
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
  __syncthreads();
  if (live) {
    float off = 0.f;
    for (int g = 0; g < tg; ++g) off += tot[g * dk + c];
    for (int t = tg * len; t < tg * len + len; ++t) {
      const float b = b_s[t * bp + c] + off;
      b_s[t * bp + c] = b;
      if (t < at.n) p.cum[size_t(at.t0 + t) * (H * dk) + h * dk + c] = b;
    }
    if (tg == TG - 1) p.gam[(at.index * H + h) * dk + c] = exp2f(b_s[(kGc - 1) * bp + c]);
  }
  gc_wait<1>();
  __syncthreads();
  for (int ch = lane * 2; ch < dk; ch += 64) {
    const float2 e = *reinterpret_cast<const float2*>(b_s + (kGc - 1) * bp + ch);
#pragma unroll
    for (int i = 0; i < kGc / kGcWarps; ++i) {
      const int t = warp + kGcWarps * i;
      float2 x = gc_pair(k_lo + t * kp + ch);
      const float2 b = *reinterpret_cast<const float2*>(b_s + t * bp + ch);
      x.x *= gc_exp2(e.x - b.x);
      x.y *= gc_exp2(e.y - b.y);
      gc_split(x.x, x.y, *reinterpret_cast<uint32_t*>(k_hi + t * kp + ch), *reinterpret_cast<uint32_t*>(k_lo + t * kp + ch));
    }
  }
  gc_wait<0>();
  __syncthreads();
  // ----- U = (2^(b_C - b) k)^T V: jobs of 16 rows x 32 columns -----
  float* u = p.u + (at.index * H + h) * size_t(dk) * dv;
  const int mat = lane >> 3, mrow = lane & 7, g = lane >> 2, t4 = lane & 3;
  const int nbs = (dv + 31) / 32;
  const int steps = (at.n + 15) / 16;
  for (int job = warp; job < (dk / 16) * nbs; job += kGcWarps) {
    const int m0 = job / nbs * 16, n0 = (job % nbs) * 32, tiles = min(4, (dv - n0) / 8);  // 2 or 4: dv is a multiple of 16
    float acc[4][4] = {};
    for (int ks = 0; ks < steps; ++ks) {
      uint32_t hi[4], lo[4], v[2][4];
      const int off = (ks * 16 + (mat >> 1) * 8 + mrow) * kp + m0 + (mat & 1) * 8;
      gc_ldm_t(smem_u32(k_hi + off), hi);
      gc_ldm_t(smem_u32(k_lo + off), lo);
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (2 * i < tiles) gc_ldm_t(smem_u32(v_s + (ks * 16 + (mat & 1) * 8 + mrow) * vp + n0 + i * 16 + (mat >> 1) * 8), v[i]);
#pragma unroll
      for (int part = 0; part < 2; ++part)  // all tiles between two additions to the same one
#pragma unroll
        for (int i = 0; i < 2; ++i)
          if (2 * i < tiles) {
            gc_mma(acc[2 * i], part ? lo : hi, v[i][0], v[i][1]);
            gc_mma(acc[2 * i + 1], part ? lo : hi, v[i][2], v[i][3]);
          }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      if (nt < tiles) {
        float* d = u + size_t(m0 + g) * dv + n0 + nt * 8 + t4 * 2;
        *reinterpret_cast<float2*>(d) = make_float2(acc[nt][0], acc[nt][1]);
        *reinterpret_cast<float2*>(d + size_t(8) * dv) = make_float2(acc[nt][2], acc[nt][3]);
      }
    }
  }
}

__global__ void __launch_bounds__(128)
gla_chunk_state_kernel(const GlaChunkParams p) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z, H = p.s.H, dk = p.s.dk, dv = p.s.dv;
  const int slot = p.slot[b], r0 = p.starts[b], len = p.starts[b + 1] - r0;
  const int e = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (slot < 0 || e >= dk * dv) return;
  const int chunks = (len + kGc - 1) / kGc, row = e / dv;
  const size_t first = size_t((r0 - p.starts[0]) / kGc + b), step = size_t(H) * dk * dv;
  float* u = p.u + (first * H + h) * size_t(dk) * dv + e;
  const float* gam = p.gam + (first * H + h) * dk + row;
  float* st = p.state + (size_t(slot) * H + h) * dk * dv + e;
  float s[8];
  load8<float>(st, s);
  constexpr int kAhead = 8;
  for (int c0 = 0; c0 < chunks; c0 += kAhead) {
    float x[kAhead][8], gm[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (c0 + i < chunks) {
        load8<float>(u + (c0 + i) * step, x[i]);
        gm[i] = gam[size_t(c0 + i) * H * dk];
      }
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (c0 + i < chunks) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) gc_split(s[2 * j], s[2 * j + 1], hi[j], lo[j]);
        uint4* d = reinterpret_cast<uint4*>(u + (c0 + i) * step);
        d[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        d[1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
        for (int j = 0; j < 8; ++j) s[j] = fmaf(gm[i], s[j], x[i][j]);
      }
  }
  store8<float>(st, s);
}

struct GlaOutputSmem {
  int b, q, a, v, ss, bytes, stages;
};
__host__ __device__ inline GlaOutputSmem gc_output_smem(int dk, int dv) {
  GlaOutputSmem m{};
  m.b = 0;                                             // b [64][dk + 8] fp32, then stages of S_0: [16][dv * 4 + 16 bytes]
  const int bb = kGc * (dk + 8) * 4, stage = 16 * (dv * 4 + 16), sb = 2 * stage;
  m.stages = bb >= 4 * stage ? 4 : 2;
  m.q = m.b + (bb > sb ? bb : sb);                     // q, k [64][dk + 8] bf16, then hi, lo of 2^b q
  m.a = m.q + 2 * kGc * (dk + 8) * 2;                  // partial sums of A [64][72] fp32, then A hi, lo [64][72] bf16
  m.v = m.a + 2 * kGc * 72 * 2;                        // [64][dv + 8] bf16
  m.ss = m.v + kGc * (dv + 8) * 2;                     // [4][64] fp32
  m.bytes = m.ss + 1024;
  return m;
}

// NT: upper bound of the 8-column tiles of a warp (dv / 32)
template <int NT, bool kBonus>
__global__ void __launch_bounds__(kGcThreads, NT <= 4 ? 2 : 1)
gla_chunk_output_kernel(const GlaChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t gc_sm[];
  pdl_wait();
  GlaChunkAt at;
  if (!gc_locate(p, blockIdx.x, blockIdx.z, at)) return;
  const int h = blockIdx.y, H = p.s.H, dk = p.s.dk, dv = p.s.dv;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int mat = lane >> 3, mrow = lane & 7, g = lane >> 2, t4 = lane & 3;
  const GlaOutputSmem m = gc_output_smem(dk, dv);
  float* b_s = reinterpret_cast<float*>(gc_sm + m.b);
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.q);
  __nv_bfloat16* a_hi = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.a);
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(gc_sm + m.v);
  float* ss_s = reinterpret_cast<float*>(gc_sm + m.ss);
  const int bp = dk + 8, kp = dk + 8, vp = dv + 8, ap = 72;
  __nv_bfloat16* k_s = q_s + kGc * kp;
  __nv_bfloat16* a_lo = a_hi + kGc * ap;
  const __nv_bfloat16* rows = p.proj + size_t(at.t0) * p.s.row_stride;
  {
    const float* cum = p.cum + size_t(at.t0) * (H * dk) + h * dk;
    for (int t = warp; t < kGc; t += kGcWarps)  // rows past the end repeat the last one
      for (int c = lane * 4; c < dk; c += 128) gc_cp16(b_s + t * bp + c, cum + size_t(min(t, at.n - 1)) * (H * dk) + c);
    gc_rows<kGcWarps>(q_s, kp, rows + h * dk, p.s.row_stride, dk, at.n, warp, lane);
    gc_rows<kGcWarps>(k_s, kp, rows + (H + h) * dk, p.s.row_stride, dk, at.n, warp, lane);
    gc_rows<kGcWarps>(v_s, vp, rows + 2 * H * dk + h * dv, p.s.row_stride, dv, at.n, warp, lane);
    gc_commit();
  }
  gc_wait<0>();
  __syncthreads();
  auto b_query = [&](int t, int c) {  // b of the state that token t reads, channels c and c + 1
    if (!kBonus) return *reinterpret_cast<const float2*>(b_s + t * bp + c);
    return t ? *reinterpret_cast<const float2*>(b_s + (t - 1) * bp + c) : make_float2(0.f, 0.f);
  };
  if (kBonus) {  // diagonal of A, kept where the norm's sums go later
    for (int t = warp; t < kGc; t += kGcWarps) {
      float x = 0.f;
      for (int c = lane * 2; c < dk; c += 64) {
        const float2 q = gc_pair(q_s + t * kp + c), k = gc_pair(k_s + t * kp + c), u = *reinterpret_cast<const float2*>(p.s.bonus + h * dk + c);
        x = fmaf(q.x * k.x, u.x, fmaf(q.y * k.y, u.y, x));
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
      if (lane == 0) ss_s[t] = x * p.s.scale;
    }
    __syncthreads();
  }
  // ----- A: warp = (row block I, one half of the column blocks J <= I, even or odd 16-channel steps); the second half of the
  //       columns is taken in reverse, so that every scheduler gets short and long row blocks -----
  const int ksteps = dk / 16;
  bool wide = false;
  {
    const bool upper = warp & 4, odd = warp & 8;
    const int I = upper ? 3 - (warp & 3) : warp & 3, J0 = upper ? (I + 2) / 2 : 0, J1 = upper ? I + 1 : (I + 2) / 2;  // J0 .. J1 - 1
    float* part = reinterpret_cast<float*>(a_hi);
    float acc[2][2][4] = {};
    const float* ref = b_s + (16 * I - 1) * bp;
    for (int ks = odd; ks < ksteps && J0 < J1; ks += 2) {
      uint32_t hi[4], lo[4];
      float2 rf[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = ks * 16 + e * 8 + t4 * 2;
        rf[e] = I ? *reinterpret_cast<const float2*>(ref + c) : make_float2(0.f, 0.f);
        const float2 last = *reinterpret_cast<const float2*>(b_s + (16 * I + 15) * bp + c);
        wide = wide || rf[e].x - last.x > kGcSpan || rf[e].y - last.y > kGcSpan;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = 16 * I + r * 8 + g;
          const float2 q = gc_pair(q_s + t * kp + c), b = b_query(t, c);
          gc_split(q.x * p.s.scale * gc_exp2(b.x - rf[e].x), q.y * p.s.scale * gc_exp2(b.y - rf[e].y), hi[e * 2 + r], lo[e * 2 + r]);
        }
      }
#pragma unroll
      for (int jj = 0; jj < 2; ++jj) {
        if (J0 + jj < J1) {
          uint32_t kh[2][2], kl[2][2];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int s = 16 * (J0 + jj) + nt * 8 + g;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int c = ks * 16 + e * 8 + t4 * 2;
              const float2 k = gc_pair(k_s + s * kp + c), b = *reinterpret_cast<const float2*>(b_s + s * bp + c);
              gc_split(k.x * gc_exp2(rf[e].x - b.x), k.y * gc_exp2(rf[e].y - b.y), kh[nt][e], kl[nt][e]);
            }
          }
          gc_mma(acc[jj][0], hi, kh[0][0], kh[0][1]);
          gc_mma(acc[jj][1], hi, kh[1][0], kh[1][1]);
          gc_mma(acc[jj][0], lo, kh[0][0], kh[0][1]);
          gc_mma(acc[jj][1], lo, kh[1][0], kh[1][1]);
          gc_mma(acc[jj][0], hi, kl[0][0], kl[0][1]);
          gc_mma(acc[jj][1], hi, kl[1][0], kl[1][1]);
        }
      }
    }
    auto each = [&](auto&& f) {  // f(pair of sums, row, first column) over my blocks
#pragma unroll
      for (int jj = 0; jj < 2; ++jj)
        if (J0 + jj < J1)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int r = 0; r < 2; ++r) f(acc[jj][nt][2 * r], acc[jj][nt][2 * r + 1], 16 * I + r * 8 + g, 16 * (J0 + jj) + nt * 8 + t4 * 2);
    };
    if (odd) each([&](float x, float y, int t, int s) { *reinterpret_cast<float2*>(part + t * ap + s) = make_float2(x, y); });
    __syncthreads();
    if (!odd)
      each([&](float& x, float& y, int t, int s) {
        const float2 o = *reinterpret_cast<const float2*>(part + t * ap + s);
        x = s + kBonus <= t ? x + o.x : (kBonus && s == t ? ss_s[t] : 0.f);
        y = s + 1 + kBonus <= t ? y + o.y : (kBonus && s + 1 == t ? ss_s[t] : 0.f);
      });
    __syncthreads();
    if (!odd)
      each([&](float x, float y, int t, int s) {
        gc_split(x, y, *reinterpret_cast<uint32_t*>(a_hi + t * ap + s), *reinterpret_cast<uint32_t*>(a_lo + t * ap + s));
      });
  }
  if (__syncthreads_or(wide)) {  // diagonal blocks term by term
    for (int i = tid; i < 4 * 256; i += kGcThreads) {
      const int t = (i >> 8) * 16 + ((i >> 4) & 15), s = (i >> 8) * 16 + (i & 15);
      if (s > t) continue;
      float x = 0.f;
      if (kBonus && s == t) continue;  // as it is
      for (int c = 0; c < dk; ++c)
        x += __bfloat162float(q_s[t * kp + c]) * __bfloat162float(k_s[s * kp + c]) * gc_exp2(b_s[(t - kBonus) * bp + c] - b_s[s * bp + c]);
      x *= p.s.scale;
      const __nv_bfloat16 hi = __float2bfloat16(x);
      a_hi[t * ap + s] = hi;
      a_lo[t * ap + s] = __float2bfloat16(x - __bfloat162float(hi));
    }
    __syncthreads();
  }
  // ----- 2^b q, in the place of q and k -----
  {
    for (int t = warp; t < kGc; t += kGcWarps)
      for (int c = lane * 2; c < dk; c += 64) {
        const float2 q = gc_pair(q_s + t * kp + c), b = b_query(t, c);
        gc_split(q.x * p.s.scale * gc_exp2(b.x), q.y * p.s.scale * gc_exp2(b.y), *reinterpret_cast<uint32_t*>(q_s + t * kp + c),
                 *reinterpret_cast<uint32_t*>(k_s + t * kp + c));
      }
  }
  __syncthreads();
  // ----- O: warp = (16 tokens, every fourth 8-column tile of the values) -----
  const uint8_t* s0 = reinterpret_cast<const uint8_t*>(p.u + (at.index * H + h) * size_t(dk) * dv);
  const int spitch = dv * 4 + 16;
  const int ahead = m.stages - 1;  // stages (a power of two) in flight while one is used
  auto fetch = [&](int ks) {
    uint8_t* d = gc_sm + m.b + (ks & ahead) * 16 * spitch;
    for (int c = lane * 16; c < dv * 4; c += 512) gc_cp16(d + warp * spitch + c, s0 + (size_t(ks) * 16 + warp) * dv * 4 + c);  // 16 warps, 16 rows
  };
  for (int ks = 0; ks < ahead; ++ks) {
    if (ks < ksteps) fetch(ks);
    gc_commit();
  }
  const int mt = warp & 4 ? 3 - (warp & 3) : warp & 3, quarter = warp >> 2, tiles = (dv / 8 - quarter + 3) / 4;
  auto col = [&](int i) { return (quarter + 4 * i) * 8; };  // first column of my i-th tile
  float o[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nt][e] = 0.f;
  const int frag = (mt * 16 + (mat & 1) * 8 + mrow), fk = (mat >> 1) * 8;
  for (int ks = 0; ks <= mt; ++ks) {
    uint32_t hi[4], lo[4];
    gc_ldm(smem_u32(a_hi + frag * ap + ks * 16 + fk), hi);
    gc_ldm(smem_u32(a_lo + frag * ap + ks * 16 + fk), lo);
#pragma unroll
    for (int n0 = 0; n0 < NT; n0 += 4) {
      uint32_t v[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (n0 + 2 * i < tiles)  // a second tile past the last is the first one again, and not used
          gc_ldm_t(smem_u32(v_s + (ks * 16 + (mat & 1) * 8 + mrow) * vp + col(min(n0 + 2 * i + (mat >> 1), tiles - 1))), v[i]);
#pragma unroll
      for (int part = 0; part < 2; ++part)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (n0 + i < tiles) gc_mma(o[n0 + i], part ? lo : hi, v[i >> 1][(i & 1) * 2], v[i >> 1][(i & 1) * 2 + 1]);
    }
  }
  // gates of my places, requested while S_0 arrives
  uint32_t gate[2][NT];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = mt * 16 + r * 8 + g;
    const __nv_bfloat16* src = rows + size_t(min(t, at.n - 1)) * p.s.row_stride + 2 * H * dk + (H + h) * dv + t4 * 2;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) gate[r][nt] = nt < tiles ? *reinterpret_cast<const uint32_t*>(src + col(nt)) : 0u;
  }
  for (int ks = 0; ks < ksteps; ++ks) {
    if (ahead == 3) gc_wait<2>();
    else gc_wait<0>();
    __syncthreads();  // step ks has arrived, and everyone is done with step ks - 1
    if (ks + ahead < ksteps) fetch(ks + ahead);
    gc_commit();
    uint32_t hi[4], lo[4];
    gc_ldm(smem_u32(q_s + frag * kp + ks * 16 + fk), hi);
    gc_ldm(smem_u32(k_s + frag * kp + ks * 16 + fk), lo);
    const uint32_t st = smem_u32(gc_sm + m.b) + (ks & ahead) * 16 * spitch + ((mat & 1) * 8 + mrow) * spitch + quarter * 32 + (mat >> 1) * 16;
#pragma unroll
    for (int n0 = 0; n0 < NT; n0 += 4) {
      uint32_t s[4][4];  // hi of rows 0-7, 8-15, then lo
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (n0 + i < tiles) gc_ldm_t(st + (n0 + i) * 128, s[i]);
#pragma unroll
      for (int part = 0; part < 3; ++part)  // all tiles between two additions to the same one
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (n0 + i < tiles) gc_mma(o[n0 + i], part == 1 ? lo : hi, s[i][part == 2 ? 2 : 0], s[i][part == 2 ? 3 : 1]);
    }
  }
  // ----- norm over the head's value channels, gate -----
  float sq[2] = {0.f, 0.f};
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    if (nt < tiles) {
      sq[0] += o[nt][0] * o[nt][0] + o[nt][1] * o[nt][1];
      sq[1] += o[nt][2] * o[nt][2] + o[nt][3] * o[nt][3];
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 1);
    sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 2);
    if (t4 == 0) ss_s[quarter * kGc + mt * 16 + r * 8 + g] = sq[r];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = mt * 16 + r * 8 + g;
    if (t >= at.n) continue;
    const float f = rsqrtf((ss_s[t] + ss_s[kGc + t] + ss_s[2 * kGc + t] + ss_s[3 * kGc + t]) * p.s.inv_dv + p.s.eps);
    __nv_bfloat16* y = p.y + (size_t(at.t0 + t) * H + h) * dv;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      if (nt < tiles) {
        const int c = col(nt) + t4 * 2;
        const float2 gt = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[r][nt])), w = *reinterpret_cast<const float2*>(p.norm_w + h * p.s.norm_stride + c);
        *reinterpret_cast<__nv_bfloat162*>(y + c) =
            __floats2bfloat162_rn(o[nt][2 * r] * f * w.x * gc_silu(gt.x), o[nt][2 * r + 1] * f * w.y * gc_silu(gt.y));
      }
    }
  }
}

template <int NT, bool kBonus>
int launch_gla_output(const GlaChunkParams& p, dim3 grid, cudaStream_t stream) {
  const int smem = gc_output_smem(p.s.dk, p.s.dv).bytes;
  static int allowed = 0;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(gla_chunk_output_kernel<NT, kBonus>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  return launch_kernel(gla_chunk_output_kernel<NT, kBonus>, grid, dim3(kGcThreads), smem, stream, p) == cudaSuccess ? 0 : -7;
}

}  // namespace
}  // namespace mfq

using namespace mfq;

// Portions of B sequences (tokens starts[b] .. starts[b + 1] - 1 of proj and y), longest `max_q`.  With chunks = T / 64 + B, T the
// tokens of all portions: cum [tokens of proj, H dk], u [chunks, H, dk, dv] and gam [chunks, H, dk] are fp32 scratch.
// Returns -5 for sizes that do not fit (callers use the token-by-token kernel).
extern "C" int mfq_gla_chunk(const void* proj, const void* w2, const float* bias, const float* norm_w, void* y, float* state,
                             const int* slot, const int* starts, float* cum, float* u, float* gam, int B, int max_q, int H, int dk, int dv,
                             int real_dv, int rank, int row_stride, float scale, float inv_tau, float eps, int decay, int norm_stride,
                             const float* bonus, cudaStream_t stream) {
  if (decay < kGlaSigmoid || decay > kGlaExp || (norm_stride && norm_stride != dv)) return -1;
  if (B <= 0 || B > 65535 || max_q <= 0 || H <= 0 || H > 65535 || dk <= 0 || dv <= 0 || dk % 16 || dv % 16 || rank <= 0 || rank % 8) return -1;
  if (real_dv <= 0 || real_dv > dv || row_stride < 2 * H * (dk + dv) + rank || row_stride % 8) return -1;
  const int local = gc_local_smem(dk, dv, rank).bytes;
  if (rank % 16 || dk > kGcMaxDk || dv > kGcMaxDv || local > 227 * 1024 || gc_output_smem(dk, dv).bytes > 227 * 1024) return -5;
  const GlaChunkParams p{GlaShape{H, dk, dv, rank, row_stride, scale, inv_tau, 1.f / float(real_dv), eps, decay, norm_stride, bonus}, static_cast<const __nv_bfloat16*>(proj),
                         static_cast<const __nv_bfloat16*>(w2), bias, norm_w, static_cast<__nv_bfloat16*>(y), starts, slot, state, cum, u, gam};
  const dim3 grid((max_q + kGc - 1) / kGc, H, B);
  static int allowed = 0;
  if (local > allowed) {
    if (cudaFuncSetAttribute(gla_chunk_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, local) != cudaSuccess) return -6;
    allowed = local;
  }
  launch_kernel(gla_chunk_local_kernel, grid, dim3(kGcThreads), local, stream, p);
  launch_kernel(gla_chunk_state_kernel, dim3((dk * dv / 8 + 127) / 128, H, B), dim3(128), 0, stream, p);
  auto output = [&](auto with_bonus) {
    constexpr bool kBonus = decltype(with_bonus)::value;
    return dv <= 128 ? launch_gla_output<4, kBonus>(p, grid, stream)
                     : dv <= 256 ? launch_gla_output<8, kBonus>(p, grid, stream) : launch_gla_output<16, kBonus>(p, grid, stream);
  };
  const int rc = bonus ? output(std::true_type{}) : output(std::false_type{});
  return rc == 0 && cudaGetLastError() == cudaSuccess ? 0 : (rc ? rc : -7);
}

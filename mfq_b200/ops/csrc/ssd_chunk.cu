// State-space recurrence over prompt portions in chunks of 64 or 128 tokens, bf16 (see ssd.cuh for the recurrence).
//
// With b_t the running sum of g inside a chunk, S_0 the state before it and L its length,
//     y_t = 2^b_t (C_t S_0) + sum_{s <= t} (C_t . B_s) 2^(b_t - b_s) dt_s x_s + skip x_t
//     S_L = 2^b_L S_0 + U,       U = sum_s B_s (2^(b_L - b_s) dt_s x_s)^T
// so all that is sequential is one multiply-add per state element and chunk.  Three kernels; a CTA takes one chunk and a run of heads of
// one group, whose B and C it reads once, and goes through their columns 64 at a time:
//
//   ssd_chunk_local    running sums b, and U
//   ssd_chunk_state    a thread per eight state elements: replaces every U by the S_0 of its chunk, advances the state
//   ssd_chunk_output   C B^T once (in accumulators: a warp owns 16 tokens), then per item decays, (C B^T) x and C S_0; the next item's x
//                      and S_0 arrive meanwhile where shared memory has room for two
//
// Exponents are never positive.  Precision: B, C and x are bf16 as they come; every fp32 operand (decayed scores, decayed x, S_0) is split
// into two bf16 numbers, so sums are kept to fp32 level on bf16 tensor cores.
#include "chunk_ops.cuh"
#include "ssd.cuh"

namespace mfq {
namespace {

constexpr int kScCols = 64, kScPitch = kScCols + 8, kScState = kScCols * 4 + 16;  // columns of an item; pitch of x; bytes of a row of S_0

struct SsdChunkParams {
  SsdShape s;
  const __nv_bfloat16* x;
  const __nv_bfloat16* z;
  __nv_bfloat16* y;  // [T, H P]
  float* u;          // [chunks, H, N, P] U, then S_0 as [hi x 8 | lo x 8] bf16 per eight elements
  float* gam;        // [chunks, H] 2^b_L
  int heads, stages; // heads of a CTA; buffers of the output kernel
};

// A CTA's chunk: tokens t0 .. t0 + n - 1; `index` numbers the chunks of all portions without overlap.
struct SsdChunkAt {
  int t0, n;
  size_t index;
};
template <int L>
__device__ __forceinline__ bool sc_locate(const SsdShape& s, int chunk, int b, SsdChunkAt& at) {
  const int r0 = s.starts[b], len = s.starts[b + 1] - r0;
  at.t0 = r0 + chunk * L;
  at.n = min(L, len - chunk * L);
  at.index = size_t((r0 - s.starts[0]) / L + b + chunk);
  return at.n > 0 && s.slot[b] >= 0;
}

// dt and b of every token of the chunk for heads h0 .. h0 + heads - 1 into dt_s, b_s [heads][L]; a warp per head.  Rows past the end: dt 0.
template <int L>
__device__ __forceinline__ void sc_steps(const SsdChunkParams& p, const SsdChunkAt& at, int h0, float* dt_s, float* b_s, int warp, int warps, int lane) {
  for (int i = warp; i < p.heads; i += warps) {
    const int h = h0 + i;
    const float bias = p.s.dt_bias[h], rate = p.s.rate[h] * 1.4426950408889634f;
    float run = 0.f;
    float raw[L / 32];
#pragma unroll
    for (int j = 0; j < L / 32; ++j) raw[j] = __bfloat162float(p.z[size_t(at.t0 + min(j * 32 + lane, at.n - 1)) * p.s.z_stride + h]);
#pragma unroll
    for (int j = 0; j < L / 32; ++j) {
      const int t = j * 32 + lane;
      const float dt = t < at.n ? ssd_softplus(raw[j] + bias) : 0.f;
      float sum = dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
      }
      sum += run;
      run = __shfl_sync(0xffffffffu, sum, 31);
      dt_s[i * L + t] = dt;
      b_s[i * L + t] = -rate * sum;
    }
  }
}

// `rows` rows of `width` bf16 (a multiple of 16) to shared memory; rows from `n` on are zeros.
__device__ __forceinline__ void sc_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int stride, int width, int n, int rows, int tid, int threads) {
  const int per = width / 8;
  for (int i = tid; i < rows * per; i += threads) {
    const int t = i / per, c = (i - t * per) * 8;
    if (t < n) gc_cp16(dst + t * pitch + c, src + size_t(t) * stride + c);
    else *reinterpret_cast<uint4*>(dst + t * pitch + c) = make_uint4(0, 0, 0, 0);
  }
}

template <int L>
int sc_local_smem(int N, int heads) { return L * (N + 8) * 2 + 2 * L * kScPitch * 2 + 2 * heads * L * 4; }
template <int L>
int sc_output_smem(int N, int heads, int stages) { return 2 * L * (N + 8) * 2 + stages * (L * kScPitch * 2 + N * kScState) + 2 * heads * L * 4; }

constexpr int kScThreads = 256;

template <int L>
__global__ void __launch_bounds__(kScThreads)
ssd_chunk_local_kernel(const SsdChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t sc_sm[];
  pdl_wait();
  SsdChunkAt at;
  if (!sc_locate<L>(p.s, blockIdx.x, blockIdx.z, at)) return;
  const int H = p.s.H, N = p.s.N, P = p.s.P, h0 = blockIdx.y * p.heads, grp = h0 / (H / p.s.groups);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mat = lane >> 3, mrow = lane & 7, g = lane >> 2, t4 = lane & 3;
  const int np = N + 8, blocks = (P + kScCols - 1) / kScCols;
  __nv_bfloat16* b_m = reinterpret_cast<__nv_bfloat16*>(sc_sm);  // B [L][np]
  __nv_bfloat16* x_hi = b_m + L * np;                            // [L][pitch] each
  __nv_bfloat16* x_lo = x_hi + L * kScPitch;
  float* dt_s = reinterpret_cast<float*>(x_lo + L * kScPitch);
  float* b_s = dt_s + p.heads * L;
  const __nv_bfloat16* rows = p.x + size_t(at.t0) * p.s.x_stride;
  sc_rows(b_m, np, rows + H * P + grp * N, p.s.x_stride, N, at.n, L, tid, kScThreads);
  gc_commit();
  sc_steps<L>(p, at, h0, dt_s, b_s, warp, kScThreads / 32, lane);
  gc_wait<0>();
  const int steps = (at.n + 15) / 16;
  for (int item = 0; item < p.heads * blocks; ++item) {
    const int i = item / blocks, c0 = (item - i * blocks) * kScCols, h = h0 + i, width = min(kScCols, P - c0);
    __syncthreads();  // B, dt and b are there; everyone is done with the item before
    const float last = b_s[i * L + L - 1];
    for (int v = tid; v < steps * 16 * (kScCols / 8); v += kScThreads) {
      const int t = v / (kScCols / 8), c = (v % (kScCols / 8)) * 8;
      float a[8] = {};
      if (t < at.n && c < width) load8<__nv_bfloat16>(rows + size_t(t) * p.s.x_stride + h * P + c0 + c, a);
      const float f = dt_s[i * L + t] * gc_exp2(last - b_s[i * L + t]);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) gc_split(a[2 * j] * f, a[2 * j + 1] * f, hi[j], lo[j]);
      *reinterpret_cast<uint4*>(x_hi + t * kScPitch + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(x_lo + t * kScPitch + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    if (tid == 0 && c0 == 0) p.gam[at.index * H + h] = gc_exp2(last);
    __syncthreads();
    float* u = p.u + (at.index * H + h) * size_t(N) * P + c0;
    for (int m0 = warp * 16; m0 < N; m0 += kScThreads / 2) {
      float acc[8][4] = {};
      for (int ks = 0; ks < steps; ++ks) {
        uint32_t a[4];
        gc_ldm_t(smem_u32(b_m + (ks * 16 + (mat >> 1) * 8 + mrow) * np + m0 + (mat & 1) * 8), a);
        const int off = (ks * 16 + (mat & 1) * 8 + mrow) * kScPitch + (mat >> 1) * 8;
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            if (n * 16 < width) {
              uint32_t v[4];
              gc_ldm_t(smem_u32((part ? x_lo : x_hi) + off + n * 16), v);
              gc_mma(acc[2 * n], a, v[0], v[1]);
              gc_mma(acc[2 * n + 1], a, v[2], v[3]);
            }
          }
      }
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        if (n * 8 < width) {
          float* d = u + size_t(m0 + g) * P + n * 8 + t4 * 2;
          *reinterpret_cast<float2*>(d) = make_float2(acc[n][0], acc[n][1]);
          *reinterpret_cast<float2*>(d + size_t(8) * P) = make_float2(acc[n][2], acc[n][3]);
        }
      }
    }
  }
}

template <int L>
__global__ void __launch_bounds__(128)
ssd_chunk_state_kernel(const SsdChunkParams p) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z, H = p.s.H, size = p.s.N * p.s.P;
  const int slot = p.s.slot[b], r0 = p.s.starts[b], len = p.s.starts[b + 1] - r0;
  const int e = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (slot < 0 || e >= size) return;
  const int chunks = (len + L - 1) / L;
  const size_t first = size_t((r0 - p.s.starts[0]) / L + b), step = size_t(H) * size;
  float* u = p.u + (first * H + h) * size + e;
  const float* gam = p.gam + first * H + h;
  float* st = p.s.state + (size_t(slot) * H + h) * size + e;
  float s[8];
  load8<float>(st, s);
  constexpr int kAhead = 8;
  for (int c0 = 0; c0 < chunks; c0 += kAhead) {
    float x[kAhead][8], gm[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (c0 + i < chunks) {
        load8<float>(u + (c0 + i) * step, x[i]);
        gm[i] = gam[size_t(c0 + i) * H];
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

// A warp per 16 tokens.
template <int L>
__global__ void __launch_bounds__(L * 2)
ssd_chunk_output_kernel(const SsdChunkParams p) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t sc_sm[];
  pdl_wait();
  SsdChunkAt at;
  if (!sc_locate<L>(p.s, blockIdx.x, blockIdx.z, at)) return;
  constexpr int kThreads = L * 2, kBlocks = L / 16;
  const int H = p.s.H, N = p.s.N, P = p.s.P, h0 = blockIdx.y * p.heads, grp = h0 / (H / p.s.groups);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mat = lane >> 3, mrow = lane & 7, g = lane >> 2, t4 = lane & 3;
  const int np = N + 8, blocks = (P + kScCols - 1) / kScCols, items = p.heads * blocks;
  const int x_bytes = L * kScPitch * 2, s_bytes = N * kScState;
  __nv_bfloat16* c_m = reinterpret_cast<__nv_bfloat16*>(sc_sm);  // C [L][np]
  __nv_bfloat16* b_m = c_m + L * np;                             // B [L][np]
  uint8_t* ring = reinterpret_cast<uint8_t*>(b_m + L * np);      // stages of x [L][pitch], S_0 [N][kScState bytes]
  float* dt_s = reinterpret_cast<float*>(ring + p.stages * (x_bytes + s_bytes));
  float* b_s = dt_s + p.heads * L;
  const __nv_bfloat16* rows = p.x + size_t(at.t0) * p.s.x_stride;
  auto fetch = [&](int item) {
    const int i = item / blocks, c0 = (item - i * blocks) * kScCols, h = h0 + i, width = min(kScCols, P - c0);
    uint8_t* d = ring + (p.stages > 1 ? item & 1 : 0) * (x_bytes + s_bytes);
    sc_rows(reinterpret_cast<__nv_bfloat16*>(d), kScPitch, rows + h * P + c0, p.s.x_stride, width, at.n, L, tid, kThreads);
    const uint8_t* src = reinterpret_cast<const uint8_t*>(p.u + (at.index * H + h) * size_t(N) * P + c0);
    const int per = width / 4;
    for (int v = tid; v < N * per; v += kThreads) {
      const int r = v / per, c = (v - r * per) * 16;
      gc_cp16(d + x_bytes + r * kScState + c, src + size_t(r) * P * 4 + c);
    }
  };
  sc_rows(c_m, np, rows + H * P + (p.s.groups + grp) * N, p.s.x_stride, N, at.n, L, tid, kThreads);
  sc_rows(b_m, np, rows + H * P + grp * N, p.s.x_stride, N, at.n, L, tid, kThreads);
  gc_commit();
  fetch(0);
  gc_commit();
  sc_steps<L>(p, at, h0, dt_s, b_s, warp, kThreads / 32, lane);
  gc_wait<1>();
  __syncthreads();
  // row blocks of the two warps of a scheduler add up to the same work
  const int mt = L == 128 && warp >= 4 ? 11 - warp : warp, ksteps = N / 16;
  const bool live = mt * 16 < at.n;
  const uint32_t c_frag = smem_u32(c_m + (mt * 16 + (mat & 1) * 8 + mrow) * np + (mat >> 1) * 8);
  float s[kBlocks][2][4];  // C B^T of my tokens and the 16 tokens of every block up to mine
#pragma unroll
  for (int J = 0; J < kBlocks; ++J)
#pragma unroll
    for (int e = 0; e < 8; ++e) s[J][e >> 2][e & 3] = 0.f;
  if (live)
    for (int ks = 0; ks < ksteps; ++ks) {
      uint32_t a[4];
      gc_ldm(c_frag + ks * 32, a);
#pragma unroll
      for (int J = 0; J < kBlocks; ++J)
        if (J <= mt) {
          uint32_t k[4];
          gc_ldm(smem_u32(b_m + (J * 16 + (mat >> 1) * 8 + mrow) * np + ks * 16 + (mat & 1) * 8), k);
          gc_mma(s[J][0], a, k[0], k[1]);
          gc_mma(s[J][1], a, k[2], k[3]);
        }
    }
  const int r0 = mt * 16 + g;  // my rows: r0 and r0 + 8
  for (int item = 0; item < items; ++item) {
    const int i = item / blocks, c0 = (item - i * blocks) * kScCols, h = h0 + i, width = min(kScCols, P - c0);
    if (p.stages > 1 && item + 1 < items) {
      fetch(item + 1);
      gc_commit();
      gc_wait<1>();
    } else {
      gc_wait<0>();
    }
    __syncthreads();  // the item is there
    const uint8_t* d = ring + (p.stages > 1 ? item & 1 : 0) * (x_bytes + s_bytes);
    const __nv_bfloat16* x_m = reinterpret_cast<const __nv_bfloat16*>(d);
    if (live) {
      float o[8][4] = {};
      const uint32_t st = smem_u32(d + x_bytes) + ((mat & 1) * 8 + mrow) * kScState + (mat >> 1) * 16;
      for (int ks = 0; ks < ksteps; ++ks) {  // C S_0
        uint32_t a[4];
        gc_ldm(c_frag + ks * 32, a);
#pragma unroll
        for (int n0 = 0; n0 < 8; n0 += 4) {
          uint32_t v[4][4];  // hi of rows 0-7, 8-15, then lo
#pragma unroll
          for (int n = 0; n < 4; ++n)
            if ((n0 + n) * 8 < width) gc_ldm_t(st + ks * 16 * kScState + (n0 + n) * 32, v[n]);
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int n = 0; n < 4; ++n)
              if ((n0 + n) * 8 < width) gc_mma(o[n0 + n], a, v[n][part * 2], v[n][part * 2 + 1]);
        }
      }
      const float* bt = b_s + i * L;
      const float* dt = dt_s + i * L;
      const float b0 = bt[r0], b1 = bt[r0 + 8], f0 = gc_exp2(b0), f1 = gc_exp2(b1);
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1;
      }
#pragma unroll
      for (int J = 0; J < kBlocks; ++J) {
        if (J <= mt) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int c = J * 16 + nt * 8 + t4 * 2;
            const float2 bs = *reinterpret_cast<const float2*>(bt + c), ds = *reinterpret_cast<const float2*>(dt + c);
            const float x0 = c <= r0 ? s[J][nt][0] * gc_exp2(b0 - bs.x) * ds.x : 0.f, y0 = c + 1 <= r0 ? s[J][nt][1] * gc_exp2(b0 - bs.y) * ds.y : 0.f;
            const float x1 = c <= r0 + 8 ? s[J][nt][2] * gc_exp2(b1 - bs.x) * ds.x : 0.f;
            const float y1 = c + 1 <= r0 + 8 ? s[J][nt][3] * gc_exp2(b1 - bs.y) * ds.y : 0.f;
            gc_split(x0, y0, hi[nt * 2], lo[nt * 2]);
            gc_split(x1, y1, hi[nt * 2 + 1], lo[nt * 2 + 1]);
          }
          const uint32_t xa = smem_u32(x_m + (J * 16 + (mat & 1) * 8 + mrow) * kScPitch + (mat >> 1) * 8);
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            if (n * 16 < width) {
              uint32_t v[4];
              gc_ldm_t(xa + n * 32, v);
              gc_mma(o[2 * n], hi, v[0], v[1]);
              gc_mma(o[2 * n + 1], hi, v[2], v[3]);
              gc_mma(o[2 * n], lo, v[0], v[1]);
              gc_mma(o[2 * n + 1], lo, v[2], v[3]);
            }
          }
        }
      }
      const float skip = p.s.skip[h];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = r0 + r * 8;
        if (t < at.n) {
          __nv_bfloat16* y = p.y + (size_t(at.t0 + t) * H + h) * P + c0 + t4 * 2;
#pragma unroll
          for (int n = 0; n < 8; ++n) {
            if (n * 8 < width) {
              const float2 xv = gc_pair(x_m + t * kScPitch + n * 8 + t4 * 2);
              *reinterpret_cast<__nv_bfloat162*>(y + n * 8) = __floats2bfloat162_rn(fmaf(skip, xv.x, o[n][2 * r]), fmaf(skip, xv.y, o[n][2 * r + 1]));
            }
          }
        }
      }
    }
    if (item + 1 < items) __syncthreads();  // everyone is done with the item
    if (p.stages == 1 && item + 1 < items) {
      fetch(item + 1);
      gc_commit();
    }
  }
}

template <int L>
int launch_ssd_chunk(SsdChunkParams p, int B, int max_q, int heads, cudaStream_t stream) {
  const int N = p.s.N, most = 227 * 1024;
  p.heads = heads;
  p.stages = sc_output_smem<L>(N, heads, 2) <= most ? 2 : 1;
  const int local = sc_local_smem<L>(N, heads), output = sc_output_smem<L>(N, heads, p.stages);
  if (local > most || output > most) return -5;
  static int allowed_local = 0, allowed_output = 0;
  if (local > allowed_local) {
    if (cudaFuncSetAttribute(ssd_chunk_local_kernel<L>, cudaFuncAttributeMaxDynamicSharedMemorySize, local) != cudaSuccess) return -6;
    allowed_local = local;
  }
  if (output > allowed_output) {
    if (cudaFuncSetAttribute(ssd_chunk_output_kernel<L>, cudaFuncAttributeMaxDynamicSharedMemorySize, output) != cudaSuccess) return -6;
    allowed_output = output;
  }
  const dim3 grid((max_q + L - 1) / L, p.s.H / heads, B);
  launch_kernel(ssd_chunk_local_kernel<L>, grid, dim3(kScThreads), local, stream, p);
  launch_kernel(ssd_chunk_state_kernel<L>, dim3((N * p.s.P / 8 + 127) / 128, p.s.H, B), dim3(128), 0, stream, p);
  launch_kernel(ssd_chunk_output_kernel<L>, grid, dim3(L * 2), output, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

}  // namespace
}  // namespace mfq

using namespace mfq;

// Portions of B sequences (tokens starts[b] .. starts[b + 1] - 1), longest `max_q`; operands as for mfq_ssd_recurrent, bf16.  `chunk` is 64
// or 128 tokens, `heads` (a divisor of H / groups) go to a CTA.  With chunks = T / chunk + B, T the tokens of all portions:
// u [chunks, H, N, P] and gam [chunks, H] are fp32 scratch.  Returns -5 for sizes that do not fit.
extern "C" int mfq_ssd_chunk(const void* x, const void* z, const float* dt_bias, const float* rate, const float* skip, void* y, float* state,
                             const int* slot, const int* starts, float* u, float* gam, int B, int max_q, int H, int groups, int N, int P, int x_stride,
                             int z_stride, int chunk, int heads, cudaStream_t stream) {
  if (B <= 0 || B > 65535 || max_q <= 0 || H <= 0 || H > 65535 || groups <= 0 || H % groups || N <= 0 || P <= 0 || N % 16 || P % 16 || !starts) return -1;
  if (x_stride % 8 || x_stride < H * P + 2 * groups * N || z_stride < H || heads <= 0 || (H / groups) % heads) return -1;
  const SsdChunkParams p{SsdShape{H, groups, N, P, x_stride, z_stride, dt_bias, rate, skip, starts, slot, state}, static_cast<const __nv_bfloat16*>(x),
                         static_cast<const __nv_bfloat16*>(z), static_cast<__nv_bfloat16*>(y), u, gam, heads, 1};
  if (chunk == 64) return launch_ssd_chunk<64>(p, B, max_q, heads, stream);
  return chunk == 128 ? launch_ssd_chunk<128>(p, B, max_q, heads, stream) : -1;
}

// Latent attention over unquantized pages with a sliding window: one row [c: rank | rotated key part: rot] per token serves all
// heads (pages [page][16][R], R = rank + rot; widths as stored, multiples of 16).  A query at position i sees 0 <= i - j < window.
// A head may have a sink: one more term exp(sink) of its denominator.
//
//   latent_finish   behind the projections: norm of c and rotation of the shared key part into the page; rotation of the queries'
//                   rotated part, for rows that attend in latent space and for rows that attend to expanded keys
//   latent_down     the same for the shared row alone, beside the norm of a query latent (queries then come from a product behind it)
//   latent_pages    copies the visible pages of portions into consecutive rows, from where keys and values are expanded by a product
//                   (prefill then runs window_attn_prefill.cuh on them)
//   latent_decode   bf16, attention in latent space: queries are already mapped there, the value of a token is the latent part of
//                   its row.  A CTA takes one query token, 16 or 32 heads (one or two row tiles of m16n8k16 MMAs, which share the
//                   fragments of the cache) and one KV split, eight warps, 64 tokens (four pages) per step through two cp.async
//                   stages.  Scores: warp = (page, half of the channels), summed through shared memory; softmax: two or four rows
//                   per warp; values: a warp owns every eighth 16-channel tile.
//   latent_plain    a warp per (token, head), fp32 arithmetic: the full-precision mode
#include "window_attn.cuh"

#include <cfloat>

namespace mfq {

int launch_attn_merge(const float* part, const float* part_ml, const float* sink, __nv_bfloat16* out, int B, int heads, int splits, int dv, cudaStream_t stream);

namespace {

constexpr int kLaPage = 16, kLaThreads = 256, kLaStep = 64, kLaMaxTiles = 4;

__device__ __forceinline__ void la_cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void la_ldm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void la_ldm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void la_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LatentFinishParams {
  int T, H, d, rank, rot, real_rank, real_rot, row_stride, latent_rows;  // latent_rows: rows before this one attend in latent space
  int has_kv, table_rows;
  float eps;
  const float* norm_w;  // [rank]
  const float2* rope;   // [positions][real_rot / 2]
  const int* positions;
  const int* slots;
};

// 8 channels from c of a rotated part: neighbours turn together.
template <typename T>
__device__ __forceinline__ void latent_turned(const T* src, int c, const float2* tab, int real_rot, float (&v)[8]) {
  load8<T>(src + c, v);
#pragma unroll
  for (int j = 0; j < 8; j += 2) {
    if (tab && c + j < real_rot) {
      const float2 cs = tab[(c + j) >> 1];
      const float a = v[j], b = v[j + 1];
      v[j] = a * cs.x - b * cs.y;
      v[j + 1] = b * cs.x + a * cs.y;
    }
  }
}

// dst = src / rms(src) * w over `width` stored channels, `real` of which count; a warp.
template <typename T>
__device__ __forceinline__ void latent_norm(const T* src, T* dst, const float* w, int width, int real, float eps, int lane) {
  float v[8], ss = 0.f;
  for (int c = lane * 8; c < width; c += 256) {
    load8<T>(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float f = rsqrtf(ss / float(real) + eps);
  for (int c = lane * 8; c < width; c += 256) {
    float ww[8];
    load8<T>(src + c, v);
    load8<float>(w + c, ww);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= f * ww[j];
    store8<T>(dst + c, v);
  }
}

// proj row: [H][d + rot] queries, then [rank | rot] (has_kv).  A warp per (token, query head or latent row).
template <typename T>
__global__ void __launch_bounds__(256)
latent_finish_kernel(const T* __restrict__ proj, T* __restrict__ q_latent, T* __restrict__ q_full, T* __restrict__ pages,
                     const LatentFinishParams p) {
  pdl_trigger();
  pdl_wait();
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, per = p.H + p.has_kv;
  if (item >= p.T * per) return;
  const int t = item / per, h = item - t * per, R = p.rank + p.rot, hw = p.d + p.rot;
  const float2* tab = p.rope ? p.rope + size_t(min(p.positions[t], p.table_rows - 1)) * (p.real_rot / 2) : nullptr;
  const T* row = proj + size_t(t) * p.row_stride;
  float v[8];
  if (h < p.H) {
    const T* q = row + h * hw;
    T* dst = t < p.latent_rows ? q_latent + (size_t(t) * p.H + h) * R + p.rank : q_full + (size_t(t) * p.H + h) * hw + p.d;
    for (int c = lane * 8; c < p.rot; c += 256) {
      latent_turned<T>(q + p.d, c, tab, p.real_rot, v);
      store8<T>(dst + c, v);
    }
    if (t >= p.latent_rows)
      for (int c = lane * 8; c < p.d; c += 256) {
        load8<T>(q + c, v);
        store8<T>(q_full + (size_t(t) * p.H + h) * hw + c, v);
      }
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const T* src = row + p.H * hw;
  T* dst = pages + size_t(slot) * R;  // a page is 16 consecutive rows
  latent_norm<T>(src, dst, p.norm_w, p.rank, p.real_rank, p.eps, lane);
  for (int c = lane * 8; c < p.rot; c += 256) {
    latent_turned<T>(src + p.rank, c, tab, p.real_rot, v);
    store8<T>(dst + p.rank + c, v);
  }
}

struct LatentDownParams {
  int T, q_rank, real_q_rank, rank, real_rank, rot, real_rot, row_stride, table_rows;
  float eps;
  const float* q_norm;  // [q_rank]
  const float* norm_w;  // [rank]
  const float2* rope;   // [positions][real_rot / 2]
  const int* positions;
  const int* slots;
};

// proj row: [q_rank | rank | rot].  A warp per (token, query latent or shared row).
template <typename T>
__global__ void __launch_bounds__(256)
latent_down_kernel(const T* __restrict__ proj, T* __restrict__ q_out, T* __restrict__ pages, const LatentDownParams p) {
  pdl_trigger();
  pdl_wait();
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= 2 * p.T) return;
  const int t = item >> 1;
  const T* row = proj + size_t(t) * p.row_stride;
  if (!(item & 1)) {
    latent_norm<T>(row, q_out + size_t(t) * p.q_rank, p.q_norm, p.q_rank, p.real_q_rank, p.eps, lane);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const float2* tab = p.rope ? p.rope + size_t(min(p.positions[t], p.table_rows - 1)) * (p.real_rot / 2) : nullptr;
  T* dst = pages + size_t(slot) * (p.rank + p.rot);
  latent_norm<T>(row + p.q_rank, dst, p.norm_w, p.rank, p.real_rank, p.eps, lane);
  for (int c = lane * 8; c < p.rot; c += 256) {
    float v[8];
    latent_turned<T>(row + p.q_rank + p.rank, c, tab, p.real_rot, v);
    store8<T>(dst + p.rank + c, v);
  }
}

// Page i of the copy belongs to sequence seq[i]; it is that sequence's page i - shift[seq].
__global__ void __launch_bounds__(256)
latent_pages_kernel(const uint4* __restrict__ pages, const int* __restrict__ table, const int* __restrict__ seq, const int* __restrict__ shift,
                    uint4* __restrict__ out, int vecs, int max_pages) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x, b = seq[i];
  const uint4* src = pages + size_t(table[size_t(b) * max_pages + i - shift[b]]) * vecs;
  for (int c = threadIdx.x; c < vecs; c += blockDim.x) out[size_t(i) * vecs + c] = src[c];
}

struct LatentDecodeParams {
  const __nv_bfloat16* q;   // [T, H, R]
  const __nv_bfloat16* kv;  // [pages][16][R]
  const int* table;         // [B, max_pages]
  const int* tok_seq;       // [T] row of the table, or null: row t
  const int* lens;          // [T] sequence length including the query token, minus len_add
  __nv_bfloat16* out;       // [T, H, rank]
  float* part;
  float* part_ml;
  int H, R, rank, max_pages, window, splits, len_add;
  float scale_log2;
  const float* sink;  // [H] or null
};

int la_smem(int R, int tiles) {
  const int rows = 16 * tiles;
  return (rows + 2 * kLaStep) * (R + 8) * 2 + 2 * rows * kLaStep * 4 + rows * (kLaStep + 8) * 2 + 3 * rows * 4;
}

template <int MT>
__global__ void __launch_bounds__(kLaThreads)
latent_decode_kernel(const LatentDecodeParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t la_sm[];
  constexpr int kRows = 16 * MT, kMine = 2 * MT;  // rows of the head tiles; rows whose softmax a warp computes
  const int R = p.R, pitch = R + 8;
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(la_sm);                      // [rows][pitch]
  __nv_bfloat16* kv_s = q_s + kRows * pitch;                                          // 2 stages of [64][pitch]
  float* s_part = reinterpret_cast<float*>(kv_s + 2 * kLaStep * pitch);               // [2][rows][64]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_part + 2 * kRows * kLaStep);  // [rows][72]
  float* alpha_s = reinterpret_cast<float*>(p_s + kRows * (kLaStep + 8));             // [rows], then m, l [rows] each
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mat = lane >> 3, mrow = lane & 7;
  const int t = blockIdx.x, h0 = blockIdx.y * kRows, heads = min(kRows, p.H - h0), split = blockIdx.z;
  const int pos = p.lens[t] + p.len_add - 1, lo = max(0, pos - p.window + 1);
  const int* table = p.table + size_t(p.tok_seq ? p.tok_seq[t] : t) * p.max_pages;
  const int page0 = lo / kLaPage, last = pos / kLaPage;
  const int all = pos >= 0 ? (last - page0) / 4 + 1 : 0, chunk = (all + p.splits - 1) / p.splits;  // steps
  const int step0 = split * chunk, steps = max(0, min(all, step0 + chunk) - step0);
  const int ch = R >> 3;
  int ids = 0;  // lane j: page j of the next eight steps
  auto fetch = [&](int i) {
    const int first = page0 + (step0 + i) * 4;
    if ((i & 7) == 0) ids = table[min(first + lane, last)];
    __nv_bfloat16* dst = kv_s + (i & 1) * kLaStep * pitch;
#pragma unroll
    for (int k = 0; k < 8; ++k) {  // a warp copies two rows of every page
      const int r = k * 8 + warp, page = __shfl_sync(0xffffffffu, ids, (i & 7) * 4 + (k >> 1));
      const __nv_bfloat16* src = p.kv + (size_t(page) * kLaPage + (r & 15)) * R;
      for (int c = lane; c < ch; c += 32) la_cp16(smem_u32(dst + r * pitch + c * 8), src + c * 8);
    }
  };
  for (int r = warp; r < kRows; r += 8) {
    const __nv_bfloat16* src = p.q + (size_t(t) * p.H + h0 + min(r, heads - 1)) * R;
    for (int c = lane; c < ch; c += 32) la_cp16(smem_u32(q_s + r * pitch + c * 8), src + c * 8);
  }
  if (steps > 0) fetch(0);
  la_commit();
  float o[kLaMaxTiles][MT][2][4];
#pragma unroll
  for (int i = 0; i < kLaMaxTiles; ++i)
#pragma unroll
    for (int j = 0; j < MT * 8; ++j) o[i][j >> 3][(j >> 2) & 1][j & 3] = 0.f;
  float m_run[kMine], l_run[kMine];  // of rows kMine * warp ..
#pragma unroll
  for (int e = 0; e < kMine; ++e) { m_run[e] = -FLT_MAX; l_run[e] = 0.f; }
  const int ksteps = R / 16, khalf = (ksteps + 1) / 2, tiles = p.rank / 16;
  const int page = warp & 3, k0 = warp < 4 ? 0 : khalf, k1 = warp < 4 ? khalf : ksteps;
  const uint32_t a_off = (((mat & 1) * 8 + mrow) * pitch + (mat >> 1) * 8) * 2;
  for (int i = 0; i < steps; ++i) {
    la_wait<0>();
    __syncthreads();  // step i has arrived, everyone is done with step i - 1
    if (i + 1 < steps) fetch(i + 1);
    la_commit();
    const __nv_bfloat16* kv = kv_s + (i & 1) * kLaStep * pitch;
    {
      float s[MT][2][4] = {};
      const uint32_t qa = smem_u32(q_s) + a_off;
      const uint32_t ka = smem_u32(kv + (page * 16 + (mat >> 1) * 8 + mrow) * pitch + (mat & 1) * 8);
#pragma unroll 6
      for (int ks = k0; ks < k1; ++ks) {
        uint32_t a[MT][4], b[4];
        la_ldm(ka + ks * 32, b);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) la_ldm(qa + mt * 16 * pitch * 2 + ks * 32, a[mt]);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          la_mma(s[mt][0], a[mt], b[0], b[1]);
          la_mma(s[mt][1], a[mt], b[2], b[3]);
        }
      }
      float* d = s_part + (warp >> 2) * kRows * kLaStep + page * 16 + t4 * 2;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          *reinterpret_cast<float2*>(d + (mt * 16 + g) * kLaStep + nt * 8) = make_float2(s[mt][nt][0], s[mt][nt][1]);
          *reinterpret_cast<float2*>(d + (mt * 16 + g + 8) * kLaStep + nt * 8) = make_float2(s[mt][nt][2], s[mt][nt][3]);
        }
    }
    __syncthreads();
    const int key = (page0 + (step0 + i) * 4) * kLaPage + lane * 2;
    float x[kMine], y[kMine], mx[kMine];
#pragma unroll
    for (int e = 0; e < kMine; ++e) {
      const int r = warp * kMine + e;
      const float2 a = *reinterpret_cast<const float2*>(s_part + r * kLaStep + lane * 2);
      const float2 b = *reinterpret_cast<const float2*>(s_part + (kRows + r) * kLaStep + lane * 2);
      x[e] = key >= lo && key <= pos ? (a.x + b.x) * p.scale_log2 : -FLT_MAX;
      y[e] = key + 1 >= lo && key + 1 <= pos ? (a.y + b.y) * p.scale_log2 : -FLT_MAX;
      mx[e] = fmaxf(x[e], y[e]);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1)
#pragma unroll
      for (int e = 0; e < kMine; ++e) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], off));
#pragma unroll
    for (int e = 0; e < kMine; ++e) {
      const float mn = fmaxf(m_run[e], mx[e]), al = window_exp2(m_run[e] - mn);  // the step's first page holds a visible key
      m_run[e] = mn;
      x[e] = window_exp2(x[e] - mn);
      y[e] = window_exp2(y[e] - mn);
      l_run[e] = fmaf(l_run[e], al, x[e] + y[e]);  // of my lane's keys; the lanes meet at the end
      *reinterpret_cast<__nv_bfloat162*>(p_s + (warp * kMine + e) * (kLaStep + 8) + lane * 2) = __floats2bfloat162_rn(x[e], y[e]);
      if (lane == 0) alpha_s[warp * kMine + e] = al;
    }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float al0 = alpha_s[mt * 16 + g], al1 = alpha_s[mt * 16 + g + 8];
      if (__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) {
#pragma unroll
        for (int n = 0; n < kLaMaxTiles; ++n)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            o[n][mt][nt][0] *= al0; o[n][mt][nt][1] *= al0; o[n][mt][nt][2] *= al1; o[n][mt][nt][3] *= al1;
          }
      }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        la_ldm(smem_u32(p_s + (mt * 16 + (mat & 1) * 8 + mrow) * (kLaStep + 8) + ks * 16 + (mat >> 1) * 8), pf[mt]);
#pragma unroll
      for (int n = 0; n < kLaMaxTiles; ++n) {
        const int tile = warp + 8 * n;
        if (tile < tiles) {
          uint32_t v[4];
          la_ldm_t(smem_u32(kv + (ks * 16 + (mat & 1) * 8 + mrow) * pitch + tile * 16 + (mat >> 1) * 8), v);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            la_mma(o[n][mt][0], pf[mt], v[0], v[1]);
            la_mma(o[n][mt][1], pf[mt], v[2], v[3]);
          }
        }
      }
    }
  }
  la_wait<0>();
#pragma unroll
  for (int e = 0; e < kMine; ++e) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], off);
    if (lane == 0) {
      alpha_s[kRows + warp * kMine + e] = m_run[e];
      alpha_s[2 * kRows + warp * kMine + e] = l_run[e];
    }
  }
  __syncthreads();
  const bool whole = p.splits == 1;
#pragma unroll
  for (int rr = 0; rr < 2 * MT; ++rr) {
    const int mt = rr >> 1, half = rr & 1, r = mt * 16 + g + 8 * half;
    if (r >= heads) continue;
    const size_t row = size_t(t) * p.H + h0 + r;
    float l = alpha_s[2 * kRows + r], f = 1.f;
    if (whole) {
      if (p.sink) {  // one more key, without a value
        const float m = alpha_s[kRows + r], sink = p.sink[h0 + r] * kLog2e, mt = fmaxf(m, sink);
        f = window_exp2(m - mt);
        l = fmaf(l, f, window_exp2(sink - mt));
      }
      f = l > 0.f ? f / l : 0.f;
    }
#pragma unroll
    for (int n = 0; n < kLaMaxTiles; ++n) {
      const int tile = warp + 8 * n;
      if (tile < tiles) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float a = o[n][mt][nt][2 * half] * f, b = o[n][mt][nt][2 * half + 1] * f;
          const int c = tile * 16 + nt * 8 + t4 * 2;
          if (whole) *reinterpret_cast<__nv_bfloat162*>(p.out + row * p.rank + c) = __floats2bfloat162_rn(a, b);
          else *reinterpret_cast<float2*>(p.part + (row * p.splits + split) * p.rank + c) = make_float2(a, b);
        }
      }
    }
    if (!whole && warp == 0 && t4 == 0) {
      p.part_ml[(row * p.splits + split) * 2] = alpha_s[kRows + r];
      p.part_ml[(row * p.splits + split) * 2 + 1] = l;
    }
  }
}

template <int MT>
int launch_latent_decode(const LatentDecodeParams& p, int T, cudaStream_t stream) {
  const int smem = la_smem(p.R, MT);
  if (smem > 227 * 1024) return -5;
  static int allowed = 48 * 1024;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(latent_decode_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  launch_kernel(latent_decode_kernel<MT>, dim3(T, (p.H + 16 * MT - 1) / (16 * MT), p.splits), dim3(kLaThreads), smem, stream, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

struct LatentPlainParams {
  const int* table;
  const int* tok_seq;
  const int* positions;
  int T, H, R, rank, max_pages, window;
  float scale;
  const float* sink;  // [H] or null
};

constexpr int kLaPlainMax = 1024, kLaPlainChunks = kLaPlainMax / 256;

template <typename T>
__global__ void __launch_bounds__(128)
latent_plain_kernel(const T* __restrict__ q, const T* __restrict__ kv, T* __restrict__ out, const LatentPlainParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float sq[4][kLaPlainMax];
  __shared__ float sp[4][32];
  __shared__ int srow[4][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gw = blockIdx.x * 4 + warp;
  if (gw >= p.T * p.H) return;
  const int t = gw / p.H, pos = p.positions[t], lo = max(0, pos - p.window + 1);
  const int* table = p.table + size_t(p.tok_seq[t]) * p.max_pages;
  for (int c = lane * 8; c < p.R; c += 256) {
    float x[8];
    load8<T>(q + size_t(gw) * p.R + c, x);
#pragma unroll
    for (int j = 0; j < 8; ++j) sq[warp][c + j] = x[j];
  }
  __syncwarp();
  float m = -FLT_MAX, l = 0.f, acc[kLaPlainChunks][8] = {};
  if (p.sink) {
    m = p.sink[gw - t * p.H];
    l = 1.f;
  }
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    const int key = j0 + lane;
    float s = -FLT_MAX;
    int row = 0;
    if (key <= pos) {
      row = table[key / kLaPage] * kLaPage + key % kLaPage;
      const T* k = kv + size_t(row) * p.R;
      float dot = 0.f;
      for (int c = 0; c < p.R; c += 8) {
        float x[8];
        load8<T>(k + c, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) dot = fmaf(sq[warp][c + j], x[j], dot);
      }
      s = dot * p.scale;
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx), alpha = expf(m - mn), pr = key <= pos ? expf(s - mn) : 0.f;
    m = mn;
    float sum = pr;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = l * alpha + sum;
    sp[warp][lane] = pr;
    srow[warp][lane] = row;
    __syncwarp();
    const int cnt = min(32, pos - j0 + 1);
#pragma unroll
    for (int n = 0; n < kLaPlainChunks; ++n) {
      const int c = (n * 32 + lane) * 8;
      if (c < p.rank) {
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[n][j] *= alpha;
        for (int i = 0; i < cnt; ++i) {
          float x[8];
          load8<T>(kv + size_t(srow[warp][i]) * p.R + c, x);
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[n][j] = fmaf(sp[warp][i], x[j], acc[n][j]);
        }
      }
    }
    __syncwarp();
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int n = 0; n < kLaPlainChunks; ++n) {
    const int c = (n * 32 + lane) * 8;
    if (c < p.rank) {
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[n][j] *= inv;
      store8<T>(out + size_t(gw) * p.rank + c, acc[n]);
    }
  }
}

bool la_sizes(int H, int rank, int rot) { return H > 0 && rank > 0 && rot >= 0 && rank % 16 == 0 && rot % 16 == 0; }

}  // namespace
}  // namespace mfq

using namespace mfq;

// proj [T, row_stride]: [H][d + rot] queries, then [rank | rot] if `pages` is given.  Rows before latent_rows: the rotated part of the
// queries goes to columns rank .. of q_latent [T, H, rank + rot]; the others are written whole to q_full [T, H, d + rot].
extern "C" int mfq_latent_finish(const void* proj, int row_stride, void* q_latent, void* q_full, void* pages, const int* positions,
                                 const int* slots, const float* norm_w, const float* rope, int table_rows, int T_, int H, int d, int rank,
                                 int rot, int real_rank, int real_rot, int latent_rows, float eps, int fp32, cudaStream_t stream) {
  if (T_ <= 0 || !la_sizes(H, rank, rot) || d <= 0 || d % 16 || real_rank <= 0 || real_rank > rank || real_rot % 2 || real_rot > rot) return -1;
  if (row_stride % 8 || row_stride < H * (d + rot) + (pages ? rank + rot : 0) || (real_rot && (!rope || table_rows <= 0))) return -1;
  if ((latent_rows > 0 && !q_latent) || (latent_rows < T_ && !q_full) || (pages && (!slots || !norm_w))) return -1;
  const LatentFinishParams p{T_, H, d, rank, rot, real_rank, real_rot, row_stride, latent_rows, pages ? 1 : 0, table_rows, eps, norm_w,
                             reinterpret_cast<const float2*>(real_rot ? rope : nullptr), positions, slots};
  const long long items = (long long)(T_) * (H + (pages ? 1 : 0));
  const dim3 grid(unsigned((items + 7) / 8));
  if (fp32)
    launch_kernel(latent_finish_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(proj), static_cast<float*>(q_latent),
                  static_cast<float*>(q_full), static_cast<float*>(pages), p);
  else
    launch_kernel(latent_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(proj),
                  static_cast<__nv_bfloat16*>(q_latent), static_cast<__nv_bfloat16*>(q_full), static_cast<__nv_bfloat16*>(pages), p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// proj [T, row_stride]: [q_rank | rank | rot].  q_out [T, q_rank]: the normed query latents; pages get the shared rows.
extern "C" int mfq_latent_down(const void* proj, int row_stride, void* q_out, void* pages, const int* positions, const int* slots,
                               const float* q_norm, const float* norm_w, const float* rope, int table_rows, int T_, int q_rank, int real_q_rank,
                               int rank, int real_rank, int rot, int real_rot, float eps, int fp32, cudaStream_t stream) {
  if (T_ <= 0 || T_ > (1 << 29) || !la_sizes(1, rank, rot) || q_rank <= 0 || q_rank % 16 || real_q_rank <= 0 || real_q_rank > q_rank) return -1;
  if (real_rank <= 0 || real_rank > rank || real_rot % 2 || real_rot > rot || row_stride % 8 || row_stride < q_rank + rank + rot) return -1;
  if ((real_rot && (!rope || table_rows <= 0)) || !slots || !q_norm || !norm_w) return -1;
  const LatentDownParams p{T_, q_rank, real_q_rank, rank, real_rank, rot, real_rot, row_stride, table_rows, eps, q_norm, norm_w,
                           reinterpret_cast<const float2*>(real_rot ? rope : nullptr), positions, slots};
  const dim3 grid(unsigned((2 * T_ + 7) / 8));
  if (fp32)
    launch_kernel(latent_down_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(proj), static_cast<float*>(q_out), static_cast<float*>(pages), p);
  else
    launch_kernel(latent_down_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(proj),
                  static_cast<__nv_bfloat16*>(q_out), static_cast<__nv_bfloat16*>(pages), p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// Pages of 16 rows of R bf16.  seq [count], shift [B] as in the kernel.
extern "C" int mfq_latent_pages(const void* pages, const int* table, const int* seq, const int* shift, void* out, int count, int R,
                                int max_pages, cudaStream_t stream) {
  if (count <= 0 || R <= 0 || R % 16) return -1;
  launch_kernel(latent_pages_kernel, dim3(count), dim3(256), 0, stream, static_cast<const uint4*>(pages), table, seq, shift,
                static_cast<uint4*>(out), 2 * R, max_pages);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// q [T, H, rank + rot] -> out [T, H, rank]; sequence lengths are lens[t] + len_add; part / part_ml: scratch of T * H * splits * rank and
// * 2 floats (splits > 1).
extern "C" int mfq_latent_decode(const void* q, const void* kv, const int* table, const int* tok_seq, const int* lens, int len_add, void* out,
                                 float* part, float* part_ml, int T_, int H, int rank, int rot, int max_pages, int window, float scale,
                                 int splits, const float* sink, cudaStream_t stream) {
  if (T_ <= 0 || !la_sizes(H, rank, rot) || rank > 128 * kLaMaxTiles || window <= 0 || splits < 1 || splits > 65535 || (splits > 1 && (!part || !part_ml))) return -1;
  const LatentDecodeParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(kv), table, tok_seq, lens,
                             static_cast<__nv_bfloat16*>(out), part, part_ml, H, rank + rot, rank, max_pages, window, splits, len_add, scale * kLog2e, sink};
  const bool two = H > 16 && la_smem(rank + rot, 2) <= 227 * 1024;
  const int rc = two ? launch_latent_decode<2>(p, T_, stream) : launch_latent_decode<1>(p, T_, stream);
  if (rc) return rc;
  return splits > 1 ? launch_attn_merge(part, part_ml, sink, static_cast<__nv_bfloat16*>(out), T_, H, splits, rank, stream) : 0;
}

extern "C" int mfq_latent_plain(const void* q, const void* kv, const int* table, const int* tok_seq, const int* positions, void* out, int T_,
                                int H, int rank, int rot, int max_pages, int window, float scale, const float* sink, int fp32,
                                cudaStream_t stream) {
  if (T_ <= 0 || !la_sizes(H, rank, rot) || rank + rot > kLaPlainMax || window <= 0) return -1;
  const LatentPlainParams p{table, tok_seq, positions, T_, H, rank + rot, rank, max_pages, window, scale, sink};
  const dim3 grid(unsigned(((long long)(T_) * H + 3) / 4));
  if (fp32)
    launch_kernel(latent_plain_kernel<float>, grid, dim3(128), 0, stream, static_cast<const float*>(q), static_cast<const float*>(kv),
                  static_cast<float*>(out), p);
  else
    launch_kernel(latent_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, static_cast<const __nv_bfloat16*>(q),
                  static_cast<const __nv_bfloat16*>(kv), static_cast<__nv_bfloat16*>(out), p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

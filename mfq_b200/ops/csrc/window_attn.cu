// Sliding-window attention over unquantized pages (K [page][Hk][16][maps * dk], V [page][Hk][16][dv]), one query token per
// sequence or, in the plain kernel, any number of them.  A query at position i sees the keys j with 0 <= i - j < window, and of
// the first `keep` keys every one up to i; with a chunk size it sees the keys j <= i of its own chunk instead of a window.  Outputs may
// be turned back (window_attn.cuh: ValueTurn).  With two maps (differential attention) a KV head has two key vectors and one value
// vector per token; queries are ordered [KV head][map][query head of the KV head].  With one map a head may have a score bias by
// distance and a sink (window_attn.cuh: ScoreExtra).
//
//   window_attn_decode_kernel   bf16, one query per sequence.  A CTA serves one (sequence, KV head, KV split); its four warps
//                               take alternate pages that hold visible keys through private cp.async rings.  The (up to 16)
//                               queries of the KV head are the rows of m16n8k16 MMAs: S = Q K^T, probabilities go from
//                               accumulators straight into the A operand of P V.  Queries of both maps share the rows (and the
//                               values): a row is zero on the key channels of the other map.  Warps (and splits) merge at the end.
//   window_attn_merge_kernel    sums the splits; with two maps also the normalised difference of a head's maps
//   window_attn_plain_kernel    a warp per (token, query head), fp32 arithmetic, fp32 or bf16 storage: the full-precision mode.
#include "window_attn.cuh"

#include <cfloat>

namespace mfq {

constexpr int kWinPage = 16, kWinWarps = 4;

struct WindowDecodeParams {
  const __nv_bfloat16* q;  // [B, Hq, dk]; Hq counts the queries of all maps
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;
  const int* table;     // [B, max_pages]
  const int* seq_lens;  // length including the query token
  __nv_bfloat16* out;   // [B, Hq, dv]
  float* part;          // splits > 1 or maps > 1: [B * Hq][splits][dv]
  float* part_ml;       // [B * Hq][splits][2]
  int Hq, Hk, maps, dk, dv, max_pages, window, chunk, keep, splits, head_tiles;
  ScoreCap cap;
  ScoreExtra extra;
  ValueTurn turn;
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void win_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// DK / DV: upper bounds of the stored widths of a KV head (register arrays); the widths themselves are run-time multiples of 16.
template <int DK, int DV>
struct WinCfg {
  static constexpr int kStages = 2;  // two pages per warp in flight leave room for three CTAs per SM at 128 + 128 channels
  static int stage_bytes(int dk, int dv) { return kWinPage * (dk + 8 + dv + 8) * 2; }
  static int smem_bytes(int dk, int dv) {
    const int ring = kWinWarps * kStages * stage_bytes(dk, dv), merge = kWinWarps * 16 * (dv + 2) * 4;
    return ring > merge ? ring : merge;
  }
};

template <int DK, int DV>
__global__ void __launch_bounds__(kWinWarps * 32)
window_attn_decode_kernel(const WindowDecodeParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t win_smem[];
  constexpr int kStages = WinCfg<DK, DV>::kStages;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ht = blockIdx.x % p.head_tiles, bg = blockIdx.x / p.head_tiles;
  const int b = bg / p.Hk, g = bg - b * p.Hk, split = blockIdx.y;
  const int per = p.Hq / p.Hk, heads = min(16, per - ht * 16);
  const int head0 = g * per + ht * 16;
  const int map_dk = p.dk, dk = p.maps * p.dk, dv = p.dv;  // dk: channels of a key row, all maps
  const int pos = p.seq_lens[b] - 1;
  const int lo = first_key(pos, p.window, p.chunk);
  // pages are counted over the visible ones: `kept` pages of first tokens that lie before the window, then the window's
  const int first = pos >= 0 ? lo / kWinPage : 0, kept = min((p.keep + kWinPage - 1) / kWinPage, first), skip = first - kept;
  int page0 = 0, page1 = pos >= 0 ? pos / kWinPage + 1 - skip : 0;
  {
    const int chunk = (page1 - page0 + p.splits - 1) / p.splits;
    page0 = page0 + split * chunk;
    page1 = min(page1, page0 + chunk);
  }
  const int kpitch = dk + 8, vpitch = dv + 8;  // odd multiples of 16 bytes apart modulo 128: ldmatrix without conflicts
  const int stage_bytes = kWinPage * (kpitch + vpitch) * 2;
  const uint32_t ring = smem_u32(win_smem) + warp * kStages * stage_bytes;
  const int n = max(0, (page1 - page0 - warp + kWinWarps - 1) / kWinWarps);  // my pages: page0 + warp + 4 i
  const int* table = p.table + size_t(b) * p.max_pages;
  const int kch = dk >> 3, vch = dv >> 3;
  const uint32_t kinv = (65536u + kch - 1) / kch, vinv = (65536u + vch - 1) / vch;  // row = i / chunks for i < 512
  int ids = 0;  // lane j holds the id of my page (32 block + j)
  auto fetch = [&](int i) {
    if ((i & 31) == 0) {
      const int pg = page0 + warp + kWinWarps * (i + lane);
      ids = pg < page1 ? table[pg < kept ? pg : pg + skip] : 0;
    }
    const int page = __shfl_sync(0xffffffffu, ids, i & 31);
    const uint32_t st = ring + (i % kStages) * stage_bytes;
    const __nv_bfloat16* ks = p.k + (size_t(page) * p.Hk + g) * (kWinPage * dk);
    const __nv_bfloat16* vs = p.v + (size_t(page) * p.Hk + g) * (kWinPage * dv);
    for (int c = lane; c < kWinPage * kch; c += 32) {
      const int row = (c * kinv) >> 16;
      cp_async16(st + (row * kpitch + (c - row * kch) * 8) * 2, ks + c * 8);
    }
    const uint32_t sv = st + kWinPage * kpitch * 2;
    for (int c = lane; c < kWinPage * vch; c += 32) {
      const int row = (c * vinv) >> 16;
      cp_async16(sv + (row * vpitch + (c - row * vch) * 8) * 2, vs + c * 8);
    }
  };
#pragma unroll
  for (int i = 0; i < kStages - 1; ++i) {
    if (i < n) fetch(i);
    cp_async_commit();
  }
  // query fragments: rows r0 = lane / 4 and r0 + 8 of the head tile
  const int r0 = lane >> 2, t4 = lane & 3;
  uint32_t qf[DK / 16][4];
  {
    // a row's own map covers the key channels c0 .. c0 + map_dk - 1
    const int of_map = per / p.maps;
    const int c0 = (ht * 16 + r0) / of_map * map_dk, c1 = (ht * 16 + r0 + 8) / of_map * map_dk;
    const __nv_bfloat16* q0 = p.q + (size_t(b) * p.Hq + head0 + r0) * map_dk + t4 * 2 - c0;
    const __nv_bfloat16* q1 = p.q + (size_t(b) * p.Hq + head0 + r0 + 8) * map_dk + t4 * 2 - c1;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      const bool in0 = r0 < heads && ks * 16 >= c0 && ks * 16 < c0 + map_dk;
      const bool in1 = r0 + 8 < heads && ks * 16 >= c1 && ks * 16 < c1 + map_dk;
      qf[ks][0] = in0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16) : 0u;
      qf[ks][1] = in1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16) : 0u;
      qf[ks][2] = in0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 8) : 0u;
      qf[ks][3] = in1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 8) : 0u;
    }
  }
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  float m[2] = {-FLT_MAX, -FLT_MAX}, l[2] = {0.f, 0.f};
  const float* bias[2] = {nullptr, nullptr};  // of rows r0 and r0 + 8
  float far[2] = {0.f, 0.f};
  if (p.extra.bias) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      bias[r] = p.extra.bias + size_t(head0 + min(r0 + 8 * r, heads - 1)) * (p.extra.last + 1);
      far[r] = bias[r][p.extra.last] * kLog2e;
    }
  }
  const int mat = lane >> 3, mrow = lane & 7;
  const uint32_t k_off = (((mat >> 1) * 8 + mrow) * kpitch + (mat & 1) * 8) * 2;
  const uint32_t v_off = (((mat & 1) * 8 + mrow) * vpitch + (mat >> 1) * 8) * 2;
  for (int i = 0; i < n; ++i) {
    if (i + kStages - 1 < n) fetch(i + kStages - 1);
    cp_async_commit();
    cp_async_wait<kStages - 1>();
    __syncwarp();
    const uint32_t st = ring + (i % kStages) * stage_bytes, sv = st + kWinPage * kpitch * 2;
    float s[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      if (ks * 16 < dk) {
        uint32_t kf[4];
        ldmatrix_x4(st + k_off + ks * 32, kf);
        win_mma(s[0], qf[ks], kf[0], kf[1]);
        win_mma(s[1], qf[ks], kf[2], kf[3]);
      }
    }
    const int pg = page0 + warp + kWinWarps * i;
    const int key0 = (pg < kept ? pg : pg + skip) * kWinPage + t4 * 2;
    float mx[2] = {-FLT_MAX, -FLT_MAX};
    const bool near = pos - (key0 - t4 * 2 + kWinPage - 1) < p.extra.last;  // some key of the page is nearer than the last bias
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = key0 + nt * 8 + (e & 1);
        float c = score_any(p.cap, s[nt][e]);
        if (p.extra.bias) c += near ? bias[e >> 1][min(max(pos - key, 0), p.extra.last)] * kLog2e : far[e >> 1];
        s[nt][e] = (key >= lo || key < p.keep) && key <= pos ? c : -FLT_MAX;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[nt][e]);
      }
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float mn = fmaxf(m[r], mx[r]);  // every page holds a visible key, so mn is a real score
      alpha[r] = window_exp2(m[r] - mn);
      m[r] = mn;
      l[r] *= alpha[r];
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[nt][e] = window_exp2(s[nt][e] - m[e >> 1]);  // hidden keys: exp2 of a huge negative number
        l[e >> 1] += s[nt][e];
      }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int d = 0; d < DV / 8; ++d) {
        o[d][0] *= alpha[0]; o[d][1] *= alpha[0]; o[d][2] *= alpha[1]; o[d][3] *= alpha[1];
      }
    }
    const uint32_t pf[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
    for (int d = 0; d < DV / 16; ++d) {
      if (d * 16 < dv) {
        uint32_t vf[4];
        ldmatrix_x4_trans(sv + v_off + d * 32, vf);
        win_mma(o[2 * d], pf, vf[0], vf[1]);
        win_mma(o[2 * d + 1], pf, vf[2], vf[3]);
      }
    }
    __syncwarp();  // the stage is refilled by the next round's fetch
  }
  // ----- merge the four warps (then the splits, in a second kernel) -----
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  cp_async_wait<0>();
  __syncthreads();
  float* acc = reinterpret_cast<float*>(win_smem);              // [warp][16][dv]
  float* ml = acc + kWinWarps * 16 * dv;                        // [warp][16][2]
  {
    float* a0 = acc + (warp * 16 + r0) * dv + t4 * 2;
    float* a1 = a0 + 8 * dv;
#pragma unroll
    for (int d = 0; d < DV / 8; ++d) {
      if (d * 8 < dv) {
        *reinterpret_cast<float2*>(a0 + d * 8) = make_float2(o[d][0], o[d][1]);
        *reinterpret_cast<float2*>(a1 + d * 8) = make_float2(o[d][2], o[d][3]);
      }
    }
    if (t4 == 0) {
      ml[(warp * 16 + r0) * 2] = m[0]; ml[(warp * 16 + r0) * 2 + 1] = l[0];
      ml[(warp * 16 + r0 + 8) * 2] = m[1]; ml[(warp * 16 + r0 + 8) * 2 + 1] = l[1];
    }
  }
  __syncthreads();
  for (int r = warp; r < heads; r += kWinWarps) {
    float mw[kWinWarps], mt = -FLT_MAX, lt = 0.f;
#pragma unroll
    for (int w = 0; w < kWinWarps; ++w) { mw[w] = ml[(w * 16 + r) * 2]; mt = fmaxf(mt, mw[w]); }
    const bool whole = p.splits == 1 && p.maps == 1;
    if (whole && p.extra.sink) {
      const float sink = p.extra.sink[head0 + r] * kLog2e;
      mt = fmaxf(mt, sink);
      lt = window_exp2(sink - mt);
    }
#pragma unroll
    for (int w = 0; w < kWinWarps; ++w) {
      mw[w] = window_exp2(mw[w] - mt);  // a warp without pages: l = 0, o = 0
      lt += ml[(w * 16 + r) * 2 + 1] * mw[w];
    }
    const size_t orow = size_t(b) * p.Hq + head0 + r;
    const float inv = whole ? (lt > 0.f ? 1.f / lt : 0.f) : 1.f;
    auto merged = [&](int c) {
      float x = 0.f;
#pragma unroll
      for (int w = 0; w < kWinWarps; ++w) x += acc[(w * 16 + r) * dv + c] * mw[w];
      return x * inv;
    };
    if (whole && p.turn.rope) {
      const float2* tab = p.turn.rope + size_t(min(max(pos, 0), p.turn.rows - 1)) * p.turn.half;
      for (int c = lane; c < p.turn.half; c += 32) {
        const float2 cs = tab[c];
        const float x = merged(c), y = merged(c + p.turn.half);
        p.out[orow * dv + c] = __float2bfloat16(fmaf(x, cs.x, y * cs.y));
        p.out[orow * dv + c + p.turn.half] = __float2bfloat16(fmaf(y, cs.x, -x * cs.y));
      }
      for (int c = 2 * p.turn.half + lane; c < dv; c += 32) p.out[orow * dv + c] = __float2bfloat16(merged(c));
    } else {
      for (int c = lane; c < dv; c += 32) {
        const float x = merged(c);
        if (whole) p.out[orow * dv + c] = __float2bfloat16(x);
        else p.part[(orow * p.splits + split) * dv + c] = x;
      }
    }
    if (!whole && lane == 0) {
      p.part_ml[(orow * p.splits + split) * 2] = mt;
      p.part_ml[(orow * p.splits + split) * 2 + 1] = lt;
    }
  }
}

// A CTA per (sequence, output head).  Two maps: y = a1 - lambda a2, out = scale * y / sqrt(mean(y^2) + eps).
struct WindowMergeParams {
  const float* sink;  // [heads] or null (one map)
  int splits, dv, heads, of_map, maps;  // heads: output heads; of_map: query heads per KV head
  float lambda, scale, eps, inv_d;
  ValueTurn turn;       // one map
  const int* seq_lens;  // for the turn
};

__global__ void __launch_bounds__(128)
window_attn_merge_kernel(const float* __restrict__ part, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                         const WindowMergeParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[33];
  const int b = blockIdx.x / p.heads, h = blockIdx.x - b * p.heads, g = h / p.of_map;
  constexpr int kCols = 4;  // channels threadIdx.x + 128 i: values up to 512 wide
  float y[kCols] = {};
  for (int m = 0; m < p.maps; ++m) {
    const size_t row = (size_t(b) * p.heads + g * p.of_map) * p.maps + m * p.of_map + h - g * p.of_map;
    const float* ml = part_ml + row * p.splits * 2;
    float mt = -FLT_MAX, lt = 0.f;
#pragma unroll 8
    for (int z = 0; z < p.splits; ++z) mt = fmaxf(mt, ml[z * 2]);
    if (p.sink) {
      mt = fmaxf(mt, p.sink[h] * kLog2e);
      lt = window_exp2(p.sink[h] * kLog2e - mt);
    }
    float x[kCols] = {};
#pragma unroll 4
    for (int z = 0; z < p.splits; ++z) {
      const float w = window_exp2(ml[z * 2] - mt);
      lt = fmaf(ml[z * 2 + 1], w, lt);
      const float* src = part + (row * p.splits + z) * p.dv;
#pragma unroll
      for (int i = 0; i < kCols; ++i) {
        const int c = threadIdx.x + i * 128;
        if (c < p.dv) x[i] = fmaf(src[c], w, x[i]);
      }
    }
    const float inv = (lt > 0.f ? 1.f / lt : 0.f) * (m == 0 ? 1.f : -p.lambda);
#pragma unroll
    for (int i = 0; i < kCols; ++i) y[i] = fmaf(x[i], inv, y[i]);
  }
  float f = 1.f;
  if (p.maps == 2) f = rsqrtf(dense_block_sum(y[0] * y[0] + y[1] * y[1] + y[2] * y[2] + y[3] * y[3], red) * p.inv_d + p.eps) * p.scale;
  if (p.turn.rope) {
    __shared__ float row[512];
#pragma unroll
    for (int i = 0; i < kCols; ++i) row[threadIdx.x + i * 128] = y[i];
    __syncthreads();
    const float2* tab = p.turn.rope + size_t(min(max(p.seq_lens[b] - 1, 0), p.turn.rows - 1)) * p.turn.half;
#pragma unroll
    for (int i = 0; i < kCols; ++i) {
      const int c = threadIdx.x + i * 128;
      if (c < 2 * p.turn.half) {
        const bool low = c < p.turn.half;
        const float2 cs = tab[low ? c : c - p.turn.half];
        y[i] = fmaf(y[i], cs.x, low ? row[c + p.turn.half] * cs.y : -row[c - p.turn.half] * cs.y);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kCols; ++i) {
    const int c = threadIdx.x + i * 128;
    if (c < p.dv) out[size_t(blockIdx.x) * p.dv + c] = __float2bfloat16(y[i] * f);
  }
}

int launch_attn_merge(const float* part, const float* part_ml, const float* sink, __nv_bfloat16* out, int B, int heads, int splits, int dv,
                      cudaStream_t stream) {
  const WindowMergeParams mp{sink, splits, dv, heads, heads, 1, 0.f, 1.f, 0.f, 0.f, ValueTurn{}, nullptr};
  launch_kernel(window_attn_merge_kernel, dim3(B * heads), dim3(128), 0, stream, part, part_ml, out, mp);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

template <int DK, int DV>
static int launch_window_decode(const WindowDecodeParams& p, const WindowMergeParams& mp, int B, cudaStream_t stream) {
  const int smem = WinCfg<DK, DV>::smem_bytes(p.dk * p.maps, p.dv);
  static int allowed = 0;
  if (smem > allowed) {
    if (cudaFuncSetAttribute(window_attn_decode_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -6;
    allowed = smem;
  }
  launch_kernel(window_attn_decode_kernel<DK, DV>, dim3(B * p.Hk * p.head_tiles, p.splits), dim3(kWinWarps * 32), smem, stream, p);
  if (p.splits > 1 || p.maps > 1)
    launch_kernel(window_attn_merge_kernel, dim3(B * mp.heads), dim3(128), 0, stream, p.part, p.part_ml, p.out, mp);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

// ---------------------------------------------------------------------------------------------
// A warp per (token, query head).
// ---------------------------------------------------------------------------------------------
struct WindowPlainParams {
  const int* positions;  // [T]
  const int* tok_seq;    // [T] row of the block table
  const int* table;
  int T, Hq, Hk, maps, dk, dv, max_pages, window, chunk, keep;
  float scale, cap;
  ScoreExtra extra;
};

template <typename T>
__global__ void __launch_bounds__(128)
window_attn_plain_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ out, const WindowPlainParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ __align__(16) float sq[4][256];
  __shared__ float sp[4][32];
  __shared__ int spage[4][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gw = blockIdx.x * 4 + warp;
  if (gw >= p.T * p.Hq) return;
  const int t = gw / p.Hq, h = gw - t * p.Hq, per = p.Hq / p.Hk, g = h / per, map = (h - g * per) / (per / p.maps);
  const int pos = p.positions[t], lo = first_key(pos, p.window, p.chunk), kept = min(p.keep, lo), skip = lo - kept;
  const int* table = p.table + size_t(p.tok_seq[t]) * p.max_pages;
  if (lane * 8 < p.dk) {
    float x[8];
    load8<T>(q + (size_t(t) * p.Hq + h) * p.dk + lane * 8, x);
#pragma unroll
    for (int j = 0; j < 8; ++j) sq[warp][lane * 8 + j] = x[j];
  }
  __syncwarp();
  float m = -FLT_MAX, l = 0.f, acc[8] = {};
  if (p.extra.sink) {  // one more key, without a value
    m = p.extra.sink[h];
    l = 1.f;
  }
  for (int j0 = 0; j0 <= pos - skip; j0 += 32) {  // over the visible keys: the kept ones before the window, then the window
    const int key = j0 + lane < kept ? j0 + lane : j0 + lane + skip;
    float s = -FLT_MAX;
    int page = 0;
    if (key <= pos) {
      page = table[key / kWinPage];
      const T* kr = k + (((size_t(page) * p.Hk + g) * kWinPage + key % kWinPage) * p.maps + map) * p.dk;
      float dot = 0.f;
      for (int c = 0; c < p.dk; c += 8) {
        float x[8];
        load8<T>(kr + c, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) dot = fmaf(sq[warp][c + j], x[j], dot);
      }
      s = dot * p.scale;
      if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
      if (p.extra.bias) s += p.extra.bias[size_t(h) * (p.extra.last + 1) + min(pos - key, p.extra.last)];
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx), alpha = expf(m - mn);
    m = mn;
    const float pr = key <= pos ? expf(s - mn) : 0.f;
    float sum = pr;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = l * alpha + sum;
    sp[warp][lane] = pr;
    spage[warp][lane] = page;
    __syncwarp();
    if (lane * 8 < p.dv) {
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] *= alpha;
      const int cnt = min(32, pos - skip - j0 + 1);
      for (int i = 0; i < cnt; ++i) {
        float x[8];
        const int key_i = j0 + i < kept ? j0 + i : j0 + i + skip;
        load8<T>(v + ((size_t(spage[warp][i]) * p.Hk + g) * kWinPage + key_i % kWinPage) * p.dv + lane * 8, x);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = fmaf(sp[warp][i], x[j], acc[j]);
      }
    }
    __syncwarp();
  }
  if (lane * 8 < p.dv) {
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] *= inv;
    store8<T>(out + (size_t(t) * p.Hq + h) * p.dv + lane * 8, acc);
  }
}

}  // namespace mfq

using namespace mfq;

// One query token per sequence, bf16; Hq counts the queries of all maps.  part / part_ml: scratch of B * Hq * splits * dv and * 2
// floats (splits > 1 or maps > 1).  Two maps: out [B, Hq / 2, dv] is the normalised difference (see the merge kernel; `d` real
// value channels).
extern "C" int mfq_window_attn_decode(const void* q, const void* k, const void* v, const int* table, const int* seq_lens, void* out,
                                      float* part, float* part_ml, int B, int Hq, int Hk, int maps, int dk, int dv, int max_pages, int window,
                                      int chunk, int keep, float scale, float cap, int splits, float lambda, float out_scale, float eps, int d,
                                      const float* bias, int bias_last, const float* sink, const float* turn, int turn_d, int turn_rows,
                                      cudaStream_t stream) {
  if (chunk < 0 || (turn && (maps > 1 || turn_d <= 0 || turn_d % 2 || turn_d > dv || turn_rows <= 0))) return -1;
  if (B <= 0 || Hq <= 0 || Hk <= 0 || maps < 1 || maps > 2 || Hq % (Hk * maps) || dk % 16 || dv % 16 || dk <= 0 || dv <= 0) return -1;
  if ((bias || sink) && maps > 1) return -1;
  if (bias && bias_last < 0) return -1;
  if (dk * maps > 512 || dv > 256 || keep < 0 || (maps > 1 && (d <= 0 || d > dv))) return -1;
  if (window <= 0 || !(scale > 0.f) || splits < 1 || ((splits > 1 || maps > 1) && (!part || !part_ml))) return -1;
  const ValueTurn back{reinterpret_cast<const float2*>(turn), turn ? turn_d / 2 : 0, turn_rows};
  const WindowDecodeParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v),
                             table, seq_lens, static_cast<__nv_bfloat16*>(out), part, part_ml, Hq, Hk, maps, dk, dv, max_pages, window, chunk, keep,
                             splits, (Hq / Hk + 15) / 16, make_score_cap(scale, cap), ScoreExtra{bias, nullptr, sink, bias ? bias_last : 0}, back};
  const WindowMergeParams mp{sink, splits, dv, Hq / maps, Hq / Hk / maps, maps, lambda, out_scale, eps, maps > 1 ? 1.f / float(d) : 0.f, back, seq_lens};
  const int kw = dk * maps;
#define MFQ_WIN_DV(DK)                                                     \
  (dv <= 64 ? launch_window_decode<DK, 64>(p, mp, B, stream)               \
            : dv <= 128 ? launch_window_decode<DK, 128>(p, mp, B, stream) : launch_window_decode<DK, 256>(p, mp, B, stream))
  if (kw > 256) return launch_window_decode<512, 256>(p, mp, B, stream);
  return kw <= 64 ? MFQ_WIN_DV(64) : kw <= 128 ? MFQ_WIN_DV(128) : MFQ_WIN_DV(256);
#undef MFQ_WIN_DV
}

// Any number of query tokens: token t sits at positions[t] of the sequence in row tok_seq[t] of the block table.  Writes the
// output of every map.
extern "C" int mfq_window_attn_plain(const void* q, const void* k, const void* v, const int* table, const int* tok_seq,
                                     const int* positions, void* out, int T_, int Hq, int Hk, int maps, int dk, int dv, int max_pages,
                                     int window, int chunk, int keep, float scale, float cap, const float* bias, int bias_last, const float* sink,
                                     int fp32, cudaStream_t stream) {
  if (((bias || sink) && maps > 1) || (bias && bias_last < 0)) return -1;
  if (T_ <= 0 || Hq <= 0 || Hk <= 0 || maps < 1 || Hq % (Hk * maps) || dk % 8 || dv % 8 || dk > 256 || dv > 256 || window <= 0 || chunk < 0 || keep < 0)
    return -1;
  const WindowPlainParams p{positions, tok_seq, table, T_, Hq, Hk, maps, dk, dv, max_pages, window, chunk, keep, scale, cap, ScoreExtra{bias, nullptr, sink, bias ? bias_last : 0}};
  const dim3 grid(unsigned(((long long)(T_) * Hq + 3) / 4));
  if (fp32)
    launch_kernel(window_attn_plain_kernel<float>, grid, dim3(128), 0, stream, static_cast<const float*>(q), static_cast<const float*>(k),
                  static_cast<const float*>(v), static_cast<float*>(out), p);
  else
    launch_kernel(window_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, static_cast<const __nv_bfloat16*>(q),
                  static_cast<const __nv_bfloat16*>(k), static_cast<const __nv_bfloat16*>(v), static_cast<__nv_bfloat16*>(out), p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

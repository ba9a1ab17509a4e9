// Sliding-window attention of prompt portions on tcgen05 tensor cores, bf16, straight from the pages.
//
// A batch holds portions of several sequences; the keys and values of their tokens, and of everything before them, are in
// the pages already.  One CTA = (sequence, run of query tokens, KV head, map).  The tile's 128 rows are (token, query head of the
// KV head) pairs, so short portions fill it and keys are loaded once per group of heads; row r = token * heads + head, which is
// the order a 3-D TMA box {64 channels, heads, tokens} of q [T, Hq, dk] delivers.  With two maps (differential attention; heads
// ordered [KV head][map][head of the KV head]) a CTA takes one map: its half of the key row, and the shared values.  Per block of
// KB keys (KB / 16 pages, each one TMA box per 64 channels, page ids from the block table):
//   S = Q K^T      tcgen05.mma kind::f16, double-buffered in TMEM
//   P = softmax    8 warps, two threads per row; the scores' soft cap is a fused polynomial where all of a warp's scores are
//                  small against the cap, else the exact exponential form; masks only on blocks that need them
//   O_blk = P V    V as MN-major operand; folded into fp32 registers under the running maximum
// Only key blocks that some query of the tile can see are visited: the pages of the kept first tokens, then those of the window (or
// from the first query's chunk on);
// blocks count these pages without the gap between the two.  Head widths are multiples of 16 up to 256; channels past a
// width arrive as zeros (TMA fills them).  Pages past the sequence's last are replaced by the last one, so that every byte the
// tensor core reads is a number (hidden keys have weight zero, and zero times a number is zero).
//
// Keys and values lie in pages, or (token-major form) in rows of a plain [tokens, heads * (dk + dv)] buffer, 16 rows to a "page",
// for attention whose keys and values are made from something smaller just before.  kExtra: one map with a score bias by distance
// and / or a sink (ScoreExtra); the running maximum then starts at the sink and adds the head's largest bias to the largest score,
// an upper bound that serves as well as the maximum itself.
#pragma once

#include "window_attn.cuh"

#include <cfloat>

namespace mfq {

constexpr int kWpRows = 128, kWpPage = 16, kWpThreads = 64 + 8 * 32;

template <int DS, int VS, int KB>
struct WinPrefillCfg {
  static constexpr int kQBytes = DS * kWpRows * 128;
  static constexpr int kKSlab = KB * 128;               // [KB keys][64 channels] bf16
  static constexpr int kStage = (DS + VS) * kKSlab;
  static constexpr int kPBytes = (KB / 64) * kWpRows * 128;
  static constexpr int kSmem = kQBytes + 2 * kStage + kPBytes + 1024 + 256 + 6 * kWpRows * 4;
  static constexpr int kTmemCols = 2 * KB + 64 * VS <= 256 ? 256 : 512;
};

struct WindowPrefillParams {
  const int* q_starts;  // [B + 1] first row of every portion in q
  const int* seq_lens;  // [B] sequence length including the portion
  const int* table;     // [B, max_pages]
  __nv_bfloat16* out;   // [T, Hq, dv]
  int* status;
  int Hq, Hk, maps, dk, dv, max_pages, window, chunk, keep, per, tokens;  // per: query heads per KV head and map; tokens: query tokens per tile
  int page_rows, head_rows, head_cols;  // rows of K / V per page, between two heads; columns between two heads (token-major form)
  int group0;        // first (KV head, map) among the query heads
  const int* shift;  // [B] token-major form (no table): "page" of a sequence's first page
  ScoreCap cap;
  ScoreExtra extra;
};

struct WindowPrefillCall {
  const void *q, *k, *v;
  uint64_t k_rows, k_cols, k_stride, v_cols, v_stride;  // the 2-D tensors K and V are read as (elements)
  int T, B, max_q, groups;
};

template <int DS, int VS, int KB, bool kExtra>
__global__ void __launch_bounds__(kWpThreads, 1)
window_attn_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                           const __grid_constant__ CUtensorMap tmap_v, const WindowPrefillParams p) {
  using Cfg = WinPrefillCfg<DS, VS, KB>;
  constexpr int kHalf = KB / 2;      // key columns of a softmax thread
  constexpr int kOut = VS * 32;      // output channels of a softmax thread
  pdl_wait();
  const int seq = blockIdx.y, group = blockIdx.z, kvh = group / p.maps;  // group: (KV head, map)
  const int k_x = (group - kvh * p.maps) * p.dk + kvh * p.head_cols, v_x = kvh * p.head_cols;  // first key (of the map) / value channel
  const int q_group = p.group0 + group;
  const int row0 = p.q_starts[seq], q_len = p.q_starts[seq + 1] - row0;
  const int tiles = (q_len + p.tokens - 1) / p.tokens;
  if (int(blockIdx.x) >= tiles) return;
  const int tok0 = (tiles - 1 - blockIdx.x) * p.tokens;  // tokens of this tile: tok0 .. tok0 + n_tok - 1 of the portion
  const int n_tok = min(p.tokens, q_len - tok0);
  const int pos0 = p.seq_lens[seq] - q_len + tok0, pos_last = pos0 + n_tok - 1;
  const int* table = p.table ? p.table + size_t(seq) * p.max_pages : nullptr;
  const int shift = p.table ? 0 : p.shift[seq];
  const int first_page = first_key(pos0, p.window, p.chunk) / kWpPage, last_page = pos_last / kWpPage;
  const int kept = min((p.keep + kWpPage - 1) / kWpPage, first_page), skip = first_page - kept;  // pages before / not visited
  const int nblk = (pos_last - skip * kWpPage) / KB + 1;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = base;
  uint8_t* sKV = base + Cfg::kQBytes;  // stage s: K slabs, then V slabs
  uint8_t* sP = sKV + 2 * Cfg::kStage;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + Cfg::kPBytes);
  uint64_t* q_full = bars;
  uint64_t* kv_full = bars + 1;   // [2]
  uint64_t* kv_empty = bars + 3;  // [2]
  uint64_t* s_full = bars + 5;    // [2]
  uint64_t* s_empty = bars + 7;   // [2] 8 arrivals
  uint64_t* p_full = bars + 9;    // 8 arrivals
  uint64_t* pv_full = bars + 10;
  uint64_t* o_empty = bars + 11;  // 8 arrivals
  uint64_t* x_bar = bars + 12;    // 8 arrivals: row-maximum exchange
  uint64_t* l_bar = bars + 13;    // 8 arrivals: row-sum exchange
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 14);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_max = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 256);  // max [2 buffers][2 halves][128], sum [2][128]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&kv_full[i], 1); mbar_init(&kv_empty[i], 1); mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 8);
    }
    mbar_init(p_full, 8); mbar_init(pv_full, 1); mbar_init(o_empty, 8); mbar_init(x_bar, 8); mbar_init(l_bar, 8);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, Cfg::kTmemCols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // Only now may the next kernel be scheduled: a product kernel of the stream takes its tensor memory before it waits for
  // this one, and would hold what this CTA still needs if it came first.  (For the same reason the wait above precedes the
  // allocation.)
  pdl_trigger();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tO = tmem_base + 2 * KB;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tmap_q); tma_prefetch_desc(&tmap_k); tma_prefetch_desc(&tmap_v);
      mbar_expect_tx(q_full, uint32_t(DS) * p.per * p.tokens * 128u);  // boxes are always full: rows past the tensor are zeros
      for (int d = 0; d < DS; ++d)
        tma_load_3d(sQ + d * (kWpRows * 128), &tmap_q, q_full, d * 64, q_group * p.per, row0 + tok0);
      for (int j = 0; j < nblk; ++j) {
        const int s = j & 1;
        if (!mbar_wait(&kv_empty[s], ((j >> 1) & 1) ^ 1, abort_flag, p.status, kStatusTimeoutProducer)) break;
        uint8_t* k = sKV + s * Cfg::kStage;
        uint8_t* v = k + DS * Cfg::kKSlab;
        mbar_expect_tx(&kv_full[s], Cfg::kStage);
#pragma unroll 1
        for (int i = 0; i < KB / kWpPage; ++i) {
          const int nth = j * (KB / kWpPage) + i;
          const int nth_page = min(nth < kept ? nth : nth + skip, last_page), page = table ? table[nth_page] : nth_page + shift;
          const int row = page * p.page_rows + kvh * p.head_rows;
#pragma unroll
          for (int d = 0; d < DS; ++d) tma_load_2d(k + d * Cfg::kKSlab + i * (kWpPage * 128), &tmap_k, &kv_full[s], k_x + d * 64, row);
#pragma unroll
          for (int d = 0; d < VS; ++d) tma_load_2d(v + d * Cfg::kKSlab + i * (kWpPage * 128), &tmap_v, &kv_full[s], v_x + d * 64, row);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = umma_idesc(128, KB, 1, 1, 0, 0);
      constexpr uint32_t idesc_pv = umma_idesc(128, 64 * VS, 1, 1, 0, 1);
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      const int ksteps = p.dk / 16;
      auto issue_qk = [&](int j) {
        const uint32_t k_addr = smem_u32(sKV + (j & 1) * Cfg::kStage);
        for (int ks = 0; ks < ksteps; ++ks)
          umma_f16(tmem_base + (j & 1) * KB, umma_desc_k_sw128(q_addr + (ks >> 2) * (kWpRows * 128) + (ks & 3) * 32),
                   umma_desc_k_sw128(k_addr + (ks >> 2) * Cfg::kKSlab + (ks & 3) * 32), idesc_qk, ks > 0);
        tc_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, kStatusTimeoutMma) &&
                mbar_wait(&kv_full[0], 0, abort_flag, p.status, kStatusTimeoutMma);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
      }
      for (int j = 0; ok && j < nblk; ++j) {
        if (j + 1 < nblk) {
          const int s1 = (j + 1) & 1;
          ok = mbar_wait(&kv_full[s1], ((j + 1) >> 1) & 1, abort_flag, p.status, kStatusTimeoutMma) &&
               mbar_wait(&s_empty[s1], (((j + 1) >> 1) & 1) ^ 1, abort_flag, p.status, kStatusTimeoutMma);
          if (!ok) break;
          tc_fence_after();
          issue_qk(j + 1);
        }
        ok = mbar_wait(p_full, j & 1, abort_flag, p.status, kStatusTimeoutMma) &&
             mbar_wait(o_empty, (j & 1) ^ 1, abort_flag, p.status, kStatusTimeoutMma);
        if (!ok) break;
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sKV + (j & 1) * Cfg::kStage + DS * Cfg::kKSlab);
#pragma unroll
        for (int ks = 0; ks < KB / 16; ++ks)
          umma_f16(tO, umma_desc_k_sw128(p_addr + (ks >> 2) * (kWpRows * 128) + (ks & 3) * 32),
                   umma_desc_mn_sw128(v_addr + ks * 2048, Cfg::kKSlab), idesc_pv, ks > 0);
        tc_commit(pv_full);
        tc_commit(&kv_empty[j & 1]);
      }
    }
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    const int row = quarter * 32 + lane;
    const int tok = row / p.per;                 // rows past n_tok * per carry nothing
    const bool row_live = tok < n_tok;
    const int q_pos = pos0 + min(tok, n_tok - 1);
    const int lo = first_key(q_pos, p.window, p.chunk), lo_last = first_key(pos_last, p.window, p.chunk);
    const uint32_t lane_base = uint32_t(quarter * 32) << 16;
    float o[kOut];
#pragma unroll
    for (int d = 0; d < kOut; ++d) o[d] = 0.f;
    float m_run = -FLT_MAX, l_run = 0.f;  // maximum in transformed (log2) units
    const float* bias = nullptr;
    float far = 0.f, top = 0.f;
    if (kExtra) {
      const int head = q_group * p.per + row - tok * p.per;
      if (p.extra.bias) {
        bias = p.extra.bias + size_t(head) * (p.extra.last + 1);
        far = bias[p.extra.last] * kLog2e;
        top = p.extra.top[head] * kLog2e;
      }
      if (p.extra.sink) {
        m_run = p.extra.sink[head] * kLog2e;
        l_run = half == 0 ? 1.f : 0.f;
      }
    }
    bool ok = true;
    for (int j = 0; j < nblk; ++j) {
      const int sb = j & 1;
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[sb], (j >> 1) & 1, abort_flag, p.status, kStatusTimeoutEpilogue));
      if (!ok) break;
      tc_fence_after();
      // places count visited keys; the key at place n is n before the gap (n < kept pages), n + gap after it
      const int place0 = j * KB + half * kHalf, split = kept * kWpPage, gap = skip * kWpPage;
      // a mask is needed where the block holds kept pages, reaches past the FIRST query or starts before the LAST query's first key
      const bool masked = j * KB < split || j * KB + gap + KB - 1 > pos0 || j * KB + gap < lo_last;
      const uint32_t tS = tmem_base + sb * KB + lane_base + half * kHalf;
      float mx = -FLT_MAX, big = 0.f;
#pragma unroll
      for (int c = 0; c < kHalf; c += 32) {
        uint32_t r[32];
        tmem_ld_32x32(tS + c, r);
        tmem_wait_ld();
        if (!masked) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float s = __uint_as_float(r[i]);
            mx = fmaxf(mx, s);
            big = fmaxf(big, fabsf(s));
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float s = __uint_as_float(r[i]);
            const int n = place0 + c + i, key = n < split ? n : n + gap;
            const bool see = key <= q_pos && (key >= lo || key < p.keep);
            mx = fmaxf(mx, see ? s : -FLT_MAX);
            big = fmaxf(big, see ? fabsf(s) : 0.f);
          }
        }
      }
      const bool small = __all_sync(0xffffffffu, big <= p.cap.small || !row_live);
      s_max[(sb * 2 + half) * kWpRows + row] = mx;
      __syncwarp();
      if (lane == 0) mbar_arrive(x_bar);
      ok = __all_sync(0xffffffffu, mbar_wait(x_bar, j & 1, abort_flag, p.status, kStatusTimeoutEpilogue));
      if (!ok) break;
      mx = fmaxf(mx, s_max[(sb * 2 + (half ^ 1)) * kWpRows + row]);
      // the two threads of a row see the same maximum, so they agree on its transform
      const float m_new = fmaxf(m_run, mx == -FLT_MAX ? -FLT_MAX : score_any(p.cap, mx) + top);
      const float alpha = window_exp2(m_run - m_new);
      if (j > 0) {
        ok = __all_sync(0xffffffffu, mbar_wait(pv_full, (j - 1) & 1, abort_flag, p.status, kStatusTimeoutEpilogue));
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < kOut; c += 32) {
          uint32_t r[32];
          tmem_ld_32x32(tO + lane_base + half * kOut + c, r);
          tmem_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c + i] = (o[c + i] + __uint_as_float(r[i])) * alpha;
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(o_empty);
      }
      l_run *= alpha;
      m_run = m_new;
      float psum = 0.f;
      // columns half * kHalf + c .. : 64-key slabs of 128 bytes per row, 16-byte chunks XORed with row % 8
#pragma unroll
      for (int c = 0; c < kHalf; c += 32) {
        uint32_t r[32];
        tmem_ld_32x32(tS + c, r);
        tmem_wait_ld();
        float pr[32];
        if (p.cap.out == 0.f) {
#pragma unroll
          for (int i = 0; i < 32; ++i) pr[i] = fmaf(__uint_as_float(r[i]), p.cap.scale_log2, -m_new);
        } else if (small) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float s = __uint_as_float(r[i]), t = s * s;
            const float f = fmaf(t, fmaf(t, fmaf(t, fmaf(t, p.cap.c[4], p.cap.c[3]), p.cap.c[2]), p.cap.c[1]), p.cap.c[0]);
            pr[i] = fmaf(s, f, -m_new);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) pr[i] = score_any(p.cap, __uint_as_float(r[i])) - m_new;
        }
        if (kExtra) {
          if (bias != nullptr && pos0 - (j * KB + gap + KB - 1) < p.extra.last) {  // some pair is nearer than the last bias
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const int n = place0 + c + i, key = n < split ? n : n + gap;
              pr[i] = fmaf(__ldg(bias + min(max(q_pos - key, 0), p.extra.last)), kLog2e, pr[i]);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) pr[i] += far;
          }
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) pr[i] = window_exp2(pr[i]);
        if (masked) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int n = place0 + c + i, key = n < split ? n : n + gap;
            pr[i] = key <= q_pos && (key >= lo || key < p.keep) ? pr[i] : 0.f;
          }
        }
        const int col = half * kHalf + c;
        uint8_t* prow = sP + (col >> 6) * (kWpRows * 128) + row * 128;
#pragma unroll
        for (int ch = 0; ch < 4; ++ch) {
          uint32_t w[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float a = pr[ch * 8 + 2 * i], b = pr[ch * 8 + 2 * i + 1];
            psum += a + b;
            __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
            w[i] = *reinterpret_cast<uint32_t*>(&h);
          }
          const int chunk = (((col & 63) >> 3) + ch) ^ (row & 7);
          *reinterpret_cast<uint4*>(prow + chunk * 16) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
      l_run += psum;
      tc_fence_before();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) { mbar_arrive(&s_empty[sb]); mbar_arrive(p_full); }
    }
    if (ok) {
      s_max[(4 + half) * kWpRows + row] = l_run;
      __syncwarp();
      if (lane == 0) mbar_arrive(l_bar);
      ok = __all_sync(0xffffffffu, mbar_wait(l_bar, 0, abort_flag, p.status, kStatusTimeoutEpilogue)) &&
           __all_sync(0xffffffffu, mbar_wait(pv_full, (nblk - 1) & 1, abort_flag, p.status, kStatusTimeoutEpilogue));
      if (ok) {
        tc_fence_after();
        const float l_tot = l_run + s_max[(4 + (half ^ 1)) * kWpRows + row];
        const float inv = l_tot > 0.f ? 1.f / l_tot : 0.f;
        const int head = q_group * p.per + row - tok * p.per;
        __nv_bfloat16* dst = p.out + (size_t(row0 + tok0 + tok) * p.Hq + head) * p.dv + half * kOut;
#pragma unroll
        for (int c = 0; c < kOut; c += 32) {
          uint32_t r[32];
          tmem_ld_32x32(tO + lane_base + half * kOut + c, r);
          tmem_wait_ld();
          if (row_live) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              if (half * kOut + c + i < p.dv) {
                float v[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = (o[c + i + e] + __uint_as_float(r[i + e])) * inv;
                store8<__nv_bfloat16>(dst + c + i, v);
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem_base, Cfg::kTmemCols);
}

template <int DS, int VS, int KB, bool kExtra>
static int launch_window_prefill(const WindowPrefillParams& p, const WindowPrefillCall& c, cudaStream_t stream) {
  using Cfg = WinPrefillCfg<DS, VS, KB>;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, c.q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.dk, p.Hq, c.T, uint64_t(p.dk) * 2, uint64_t(p.Hq) * p.dk * 2, 64, p.per, p.tokens)) return -2;
  if (make_tmap_2d(&tk, c.k, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, c.k_rows, c.k_cols, c.k_stride * 2, kWpPage, 64)) return -3;
  if (make_tmap_2d(&tv, c.v, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, c.k_rows, c.v_cols, c.v_stride * 2, kWpPage, 64)) return -4;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(window_attn_prefill_kernel<DS, VS, KB, kExtra>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmem) != cudaSuccess) return -6;
    attr = true;
  }
  const dim3 grid((c.max_q + p.tokens - 1) / p.tokens, c.B, c.groups);
  launch_kernel(window_attn_prefill_kernel<DS, VS, KB, kExtra>, grid, dim3(kWpThreads), Cfg::kSmem, stream, tq, tk, tv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -7;
}

template <bool kExtra>
static int run_window_prefill(const WindowPrefillParams& p, const WindowPrefillCall& c, cudaStream_t stream) {
  const int ds = (p.dk + 63) / 64, vs = (p.dv + 63) / 64;
#define MFQ_WP(DS, VS, KB) return launch_window_prefill<DS, VS, KB, kExtra>(p, c, stream)
  if (ds == 1 && vs == 1) MFQ_WP(1, 1, 128);
  if (ds == 1 && vs == 2) MFQ_WP(1, 2, 128);
  if (ds == 2 && vs == 1) MFQ_WP(2, 1, 128);
  if (ds == 2 && vs == 2) MFQ_WP(2, 2, 128);
  if (ds <= 3 && vs <= 2) MFQ_WP(3, 2, 64);
  if (ds <= 2 && vs <= 4) MFQ_WP(2, 4, 64);
  MFQ_WP(4, 4, 64);
#undef MFQ_WP
}

int window_prefill_extra(const WindowPrefillParams& p, const WindowPrefillCall& c, cudaStream_t stream);  // window_attn_prefill_bias.cu

}  // namespace mfq

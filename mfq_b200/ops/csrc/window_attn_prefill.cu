// Entry points of the prefill attention kernel (window_attn_prefill.cuh).
#include "window_attn_prefill.cuh"

using namespace mfq;

// Portions of B sequences, longest `max_q` tokens.  q [T, Hq, dk] and out [T, Hq, dv] hold the tokens of all portions (rows
// q_starts[b] .. q_starts[b + 1] - 1 belong to sequence b), Hq counts the queries of all maps, `pages` is the number of pages of
// the pools.  One map may have a bias by distance (bias [Hq][bias_last + 1], bias_top [Hq] its largest per head) and a sink [Hq].
extern "C" int mfq_window_attn_prefill(const void* q, const void* k, const void* v, const int* table, const int* q_starts,
                                       const int* seq_lens, void* out, int T, int B, int max_q, int Hq, int Hk, int maps, int dk, int dv,
                                       int pages, int max_pages, int window, int chunk, int keep, float scale, float cap, const float* bias,
                                       int bias_last, const float* bias_top, const float* sink, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || B > 65535 || max_q <= 0 || Hq <= 0 || Hk <= 0 || maps < 1 || maps > 2 || Hk * maps > 65535) return -1;
  if (Hq % (Hk * maps) || Hq / (Hk * maps) > kWpRows || keep < 0) return -1;
  if (dk % 16 || dv % 16 || dk <= 0 || dv <= 0 || dk > 256 || dv > 256 || window <= 0 || chunk < 0 || !(scale > 0.f)) return -1;
  if (((bias || sink) && maps > 1) || (bias && (bias_last < 0 || !bias_top))) return -1;
  const int per = Hq / (Hk * maps);
  const WindowPrefillParams p{q_starts, seq_lens, table, static_cast<__nv_bfloat16*>(out), status, Hq, Hk, maps, dk, dv, max_pages, window, chunk,
                              keep, per, kWpRows / per, Hk * kWpPage, kWpPage, 0, 0, nullptr, make_score_cap(scale, cap),
                              ScoreExtra{bias, bias_top, sink, bias ? bias_last : 0}};
  const WindowPrefillCall c{q, k, v, uint64_t(pages) * Hk * kWpPage, uint64_t(maps) * dk, uint64_t(maps) * dk, uint64_t(dv), uint64_t(dv), T, B,
                            max_q, Hk * maps};
  return bias || sink ? window_prefill_extra(p, c, stream) : run_window_prefill<false>(p, c, stream);
}

// Token-major form: kv [rows, heads * (dk + dv)] holds, for `heads` heads from head0 on, the keys and values of tokens in runs of
// whole 16-row "pages"; token j of sequence b is in row (j / 16 + shift[b]) * 16 + j % 16, for every j that some query sees.  A head may have
// a sink [Hq].
extern "C" int mfq_window_attn_prefill_rows(const void* q, const void* kv, const int* shift, const int* q_starts, const int* seq_lens, void* out,
                                            int T, int B, int max_q, int Hq, int head0, int heads, int dk, int dv, int rows, int window,
                                            float scale, const float* sink, int* status, cudaStream_t stream) {
  if (T <= 0 || B <= 0 || B > 65535 || max_q <= 0 || Hq <= 0 || heads <= 0 || head0 < 0 || head0 + heads > Hq || heads > 65535) return -1;
  if (dk % 16 || dv % 16 || dk <= 0 || dv <= 0 || dk > 256 || dv > 256 || window <= 0 || !(scale > 0.f) || rows <= 0 || !shift) return -1;
  const WindowPrefillParams p{q_starts, seq_lens, nullptr, static_cast<__nv_bfloat16*>(out), status, Hq, heads, 1, dk, dv, 0, window, 0, 0, 1,
                              kWpRows, kWpPage, 0, dk + dv, head0, shift, make_score_cap(scale, 0.f), ScoreExtra{nullptr, nullptr, sink, 0}};
  const uint64_t width = uint64_t(heads) * (dk + dv);
  const WindowPrefillCall c{q, kv, static_cast<const __nv_bfloat16*>(kv) + dk, uint64_t(rows), width, width, width - dk, width, T, B, max_q, heads};
  return sink ? window_prefill_extra(p, c, stream) : run_window_prefill<false>(p, c, stream);
}

"""Latent attention over unquantized pages (``csrc/latent_attn.cu``): one row ``[c: rank | rotated key part: rot]`` per token serves
all heads of a layer, and of the layers that read its pages.

Single tokens and short portions attend in latent space: queries come mapped there (``W_uk^T q``), the value of a token is the latent
part of its row.  A head may have a sink, one more term of its denominator.  Longer bf16 portions expand the visible rows to keys and values per head (:func:`visible_rows`, a product, then
:func:`prefill_rows` on the tcgen05 kernel), which costs fewer operations per pair.
"""

from __future__ import annotations

import torch

from .dense import is_fp32
from .lib import Workspace, check, dense_lib, ptr, stream_ptr

MAX_RANK, MAX_ROW, PAGE = 512, 640, 16
EXPAND_MIN_TOKENS = 16  # a batch whose longest portion is shorter attends in latent space
EXPANDED_BYTES = 2 << 30  # most scratch for expanded keys and values; beyond, heads go in groups


def finish(proj: torch.Tensor, pages: torch.Tensor | None, positions, slots, *, heads: int, d: int, rank: int, rot: int, real_rank: int,
           real_rot: int, norm_w, rope, eps: float, latent_rows: int):
    """``proj [T, heads * (d + rot) (+ rank + rot)]``: the shared row normed, rotated and written to its page (``pages`` None: the rows
    hold queries only); returns ``(q_latent [latent_rows, heads, rank + rot]`` with the rotated part filled in, ``q [T, heads, d + rot]``
    for the other rows``)``, None where there are no such rows."""
    t = proj.shape[0]
    new = lambda n, w: torch.empty((n, heads, w), dtype=proj.dtype, device=proj.device)
    q_latent = new(latent_rows, rank + rot) if latent_rows else None
    q = new(t, d + rot) if latent_rows < t else None
    rc = dense_lib().mfq_latent_finish(ptr(proj), proj.stride(0), ptr(q_latent), ptr(q), ptr(pages), ptr(positions), ptr(slots), ptr(norm_w),
                                       ptr(rope), rope.shape[0] if rope is not None else 0, t, heads, d, rank, rot, real_rank, real_rot,
                                       latent_rows, float(eps), is_fp32(proj.dtype), stream_ptr())
    check(rc, "latent_finish")
    return q_latent, q


def down(proj: torch.Tensor, pages: torch.Tensor, positions, slots, *, q_rank: int, real_q_rank: int, rank: int, rot: int, real_rank: int, real_rot: int,
         q_norm, norm_w, rope, eps: float) -> torch.Tensor:
    """``proj [T, q_rank + rank + rot]``: the shared row as in :func:`finish`, and the normed query latents ``[T, q_rank]``, from which a
    product makes the queries (:func:`finish` without pages then turns their rotated part)."""
    t = proj.shape[0]
    out = torch.empty((t, q_rank), dtype=proj.dtype, device=proj.device)
    check(dense_lib().mfq_latent_down(ptr(proj), proj.stride(0), ptr(out), ptr(pages), ptr(positions), ptr(slots), ptr(q_norm), ptr(norm_w), ptr(rope),
                                      rope.shape[0] if rope is not None else 0, t, q_rank, real_q_rank, rank, real_rank, rot, real_rot, float(eps),
                                      is_fp32(proj.dtype), stream_ptr()), "latent_down")
    return out


def decode_splits(batch: int, heads: int, keys: int) -> int:
    """KV splits per query token and CTA (up to 32 heads) over ``keys`` visible keys: about a CTA for every SM, 128 keys each at
    least."""
    n = max(1, batch * -(-heads // 32))
    return max(1, min(148 // n if n <= 148 else 1, keys // 128, 32))


def decode(q: torch.Tensor, pages: torch.Tensor, block_table, lens, *, rank: int, window: int, scale: float, splits: int = 1,
           tok_seq: torch.Tensor | None = None, sink: torch.Tensor | None = None) -> torch.Tensor:
    """bf16 ``q [T, H, rank + rot]`` -> ``[T, H, rank]``.  ``lens`` count the query token (one row of the table per query), or with
    ``tok_seq`` (query -> row of the table) they are the queries' positions."""
    t, h, r = q.shape
    out = torch.empty((t, h, rank), dtype=q.dtype, device=q.device)
    ws = Workspace.get(q.device)
    splits = max(1, min(splits, ws.attn_acc.numel() // max(1, t * h * rank), ws.attn_ml.numel() // (2 * t * h)))
    rc = dense_lib().mfq_latent_decode(ptr(q), ptr(pages), ptr(block_table), ptr(tok_seq), ptr(lens), 0 if tok_seq is None else 1, ptr(out),
                                       ptr(ws.attn_acc), ptr(ws.attn_ml), t, h, rank, r - rank, block_table.stride(0), window, float(scale),
                                       splits, ptr(sink), stream_ptr())
    check(rc, "latent_decode", 2 if splits > 1 else 1)
    return out


def plain(q: torch.Tensor, pages: torch.Tensor, block_table, tok_seq, positions, *, rank: int, window: int, scale: float,
          sink: torch.Tensor | None = None) -> torch.Tensor:
    """The same in fp32 arithmetic: query ``t`` is at ``positions[t]`` of sequence ``tok_seq[t]``."""
    t, h, r = q.shape
    out = torch.empty((t, h, rank), dtype=q.dtype, device=q.device)
    rc = dense_lib().mfq_latent_plain(ptr(q), ptr(pages), ptr(block_table), ptr(tok_seq), ptr(positions), ptr(out), t, h, rank, r - rank,
                                      block_table.stride(0), window, float(scale), ptr(sink), is_fp32(q.dtype), stream_ptr())
    check(rc, "latent_plain")
    return out


def visible_pages(portions: list[tuple[int, int]], window: int) -> tuple[list[int], list[int]]:
    """``(sequence of every copied page, shift of every sequence)`` for portions ``(first position, tokens)``: the pages from the first
    that a query sees to the last, one sequence after the other; page p of sequence b becomes page ``p + shift[b]`` of the copy."""
    seq, shift = [], []
    for b, (start, count) in enumerate(portions):
        first, last = max(0, start - window + 1) // PAGE, (start + count - 1) // PAGE
        shift.append(len(seq) - first)
        seq += [b] * (last - first + 1)
    return seq, shift


def visible_rows(pages: torch.Tensor, block_table, seq: torch.Tensor, shift: torch.Tensor) -> torch.Tensor:
    """Copy of the visible pages ``[pages * 16, R]`` (``seq``, ``shift`` as int32 tensors)."""
    r = pages.shape[-1]
    out = torch.empty((seq.numel() * PAGE, r), dtype=pages.dtype, device=pages.device)
    check(dense_lib().mfq_latent_pages(ptr(pages), ptr(block_table), ptr(seq), ptr(shift), ptr(out), seq.numel(), r, block_table.stride(0),
                                       stream_ptr()), "latent_pages")
    return out


def prefill_rows(q: torch.Tensor, kv: torch.Tensor, shift, q_starts, seq_lens, max_q: int, *, head0: int, heads: int, dk: int, dv: int,
                 window: int, scale: float, out: torch.Tensor, sink: torch.Tensor | None = None) -> None:
    """Portions (bf16) over expanded rows: ``kv [rows, heads * (dk + dv)]`` of the heads ``head0 ..`` of ``q [T, Hq, dk]``; writes those
    heads of ``out [T, Hq, dv]``.  ``sink [Hq]``."""
    t, hq, _ = q.shape
    rc = dense_lib().mfq_window_attn_prefill_rows(ptr(q), ptr(kv), ptr(shift), ptr(q_starts), ptr(seq_lens), ptr(out), t, seq_lens.numel(), max_q,
                                                  hq, head0, heads, dk, dv, kv.shape[0], window, float(scale), ptr(sink),
                                                  ptr(Workspace.get(q.device).status), stream_ptr())
    check(rc, "window_attn_prefill_rows")

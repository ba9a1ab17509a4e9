"""Attention over unquantized pages with a sliding window and an optional score cap (``csrc/window_attn*.cu``), and the
per-head stage in front of it (``csrc/stream_ops.cu``).

A query at position ``i`` sees the keys ``j`` with ``0 <= i - j < window``; a score is ``q . k * scale``, then
``cap * tanh(score / cap)`` (``cap`` 0: no cap).  Pages: ``k [pages, Hk, 16, dk]``, ``v [pages, Hk, 16, dv]``, widths multiples
of 16 up to 256.  bf16 runs on tensor cores (one kernel for portions of prompts, one for single tokens), fp32 on a plain kernel.
"""

from __future__ import annotations

import torch

from .dense import is_fp32
from .lib import Workspace, check, dense_lib, ptr, stream_ptr

MAX_HEAD = 256
NO_WINDOW = 1 << 30


def rope_table(base: float, dims: int, positions: int, device) -> torch.Tensor:
    """``[positions, dims / 2, 2]`` fp32 (cos, sin) of ``p * base^(-2i / dims)``, evaluated in double precision."""
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)
    a = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * freq
    return torch.stack([a.cos(), a.sin()], -1).float().contiguous()


def qkv_finish(qkv: torch.Tensor, kv, positions, slots, *, heads: int, kv_heads: int, dim: int, q_norm, k_norm, rope, rot: int,
               eps: float, v_first: torch.Tensor | None = None, mix: float = 0.0) -> torch.Tensor:
    """Per-head RMS norm of q and k (over ``dim`` channels), rotation of the leading ``rot`` channels, K and V into their
    pages; returns ``q [T, heads, dk]``.  ``v_first`` (``[T, kv_heads * dv]``, rows may be strided): the cached values are
    ``(1 - mix) v + mix v_first``."""
    t = qkv.shape[0]
    dk, dv = kv.k.shape[-1], kv.v.shape[-1]
    q = torch.empty((t, heads, dk), dtype=qkv.dtype, device=qkv.device)
    rc = dense_lib().mfq_qkv_finish(ptr(qkv), qkv.stride(0), ptr(v_first), v_first.stride(0) if v_first is not None else 0, float(mix),
                                    ptr(q), ptr(kv.k), ptr(kv.v), ptr(positions), ptr(slots), ptr(q_norm), ptr(k_norm), ptr(rope),
                                    rope.shape[0] if rope is not None else 0, t, heads, kv_heads, dim, dk, dv, rot, kv.page_size,
                                    float(eps), is_fp32(qkv.dtype), stream_ptr())
    check(rc, "qkv_finish")
    return q


def decode_splits(batch: int, kv_heads: int, keys: int) -> int:
    """KV splits per (sequence, KV head) over ``keys`` visible keys, fitted to a sweep on B200 (batch 1 .. 128, windows 1024 and
    4096): a batch that leaves SMs free takes the most splits that keep the grid below 400 CTAs (at most 16, 64 keys each); one
    that comes near a wave of three CTAs per SM evens its last wave out with up to 5 splits of at least 256 keys; more is not
    split."""
    n, slots = max(1, batch * kv_heads), 148 * 3
    if n <= 200:
        return max(1, min(400 // n, keys // 64, 16))
    if n > 600:
        return 1
    choices = [s for s in range(1, 6) if s == 1 or keys // s >= 256]
    return min(choices, key=lambda s: -(-n * s // slots) * keys / s + 20 * s)


def decode(q: torch.Tensor, kv, block_table, seq_lens, *, window: int, scale: float, cap: float, splits: int = 1, out=None):
    """One query token per sequence (bf16): ``q [B, Hq, dk]`` -> ``[B, Hq, dv]``; ``seq_lens`` count the query token."""
    b, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    out = torch.empty((b, hq, dv), dtype=q.dtype, device=q.device) if out is None else out
    ws = Workspace.get(q.device)
    assert splits == 1 or (b * hq * splits * dv <= ws.attn_acc.numel() and b * hq * splits * 2 <= ws.attn_ml.numel())
    rc = dense_lib().mfq_window_attn_decode(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(seq_lens), ptr(out), ptr(ws.attn_acc),
                                            ptr(ws.attn_ml), b, hq, hk, dk, dv, block_table.stride(0), window, float(scale), float(cap),
                                            splits, stream_ptr())
    check(rc, "window_attn_decode", 2 if splits > 1 else 1)
    return out


def prefill(q: torch.Tensor, kv, block_table, q_starts, seq_lens, max_q: int, *, window: int, scale: float, cap: float, out=None):
    """Portions of several sequences (bf16): rows ``q_starts[b] .. q_starts[b + 1] - 1`` of ``q [T, Hq, dk]`` are the last
    tokens of a sequence of ``seq_lens[b]``.  ``max_q``: the longest portion (host)."""
    t, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    out = torch.empty((t, hq, dv), dtype=q.dtype, device=q.device) if out is None else out
    rc = dense_lib().mfq_window_attn_prefill(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(q_starts), ptr(seq_lens), ptr(out), t,
                                             seq_lens.numel(), max_q, hq, hk, dk, dv, kv.k.shape[0], block_table.stride(0), window,
                                             float(scale), float(cap), ptr(Workspace.get(q.device).status), stream_ptr())
    check(rc, "window_attn_prefill")
    return out


def plain(q: torch.Tensor, kv, block_table, tok_seq, positions, *, window: int, scale: float, cap: float):
    """The same in fp32 arithmetic for any mix of tokens: token ``t`` is at ``positions[t]`` of sequence ``tok_seq[t]``."""
    t, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    out = torch.empty((t, hq, dv), dtype=q.dtype, device=q.device)
    rc = dense_lib().mfq_window_attn_plain(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(tok_seq), ptr(positions), ptr(out), t, hq,
                                           hk, dk, dv, block_table.stride(0), window, float(scale), float(cap), is_fp32(q.dtype),
                                           stream_ptr())
    check(rc, "window_attn_plain")
    return out

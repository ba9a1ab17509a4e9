"""Attention over unquantized pages with a sliding window or in chunks, kept first tokens, an optional score cap and one or two maps
(``csrc/window_attn*.cu``), with one map also a score bias by distance and a sink per head, and the per-head stage in front of it (``csrc/stream_ops.cu``).

A query at position ``i`` sees the keys ``j <= i`` with ``i - j < window`` (or, with a ``chunk`` size, those of its own chunk ``i // chunk``)
or ``j < keep``; a score is ``q . k * scale``, then
``cap * tanh(score / cap)`` (``cap`` 0: no cap), then plus the head's bias for the distance ``i - j`` (:class:`DistanceBias`).  A sink
adds ``exp(sink)`` to the head's denominator.  Pages: ``k [pages, Hk, 16, maps * dk]``, ``v [pages, Hk, 16, dv]``, widths
``dk`` and ``dv`` multiples of 16 up to 256.  bf16 runs on tensor cores (one kernel for portions of prompts, one for single
tokens), fp32 on a plain kernel.

Two maps (differential attention): every query and KV head has two query / key vectors that attend on their own over the same
values; a head's output is ``rms(a1 - lambda a2) * scale`` (:class:`Difference`).  Queries are ordered ``[KV head][map][query
head of the KV head]``.

Values may carry a rotation by their position; a head's output then turns back by the query's (:class:`ValueTurn`).
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .dense import is_fp32
from .lib import Workspace, check, dense_lib, ptr, stream_ptr

MAX_HEAD = 256
NO_WINDOW = 1 << 30
MAX_BIAS_SPREAD = 60.0  # the prefill kernel adds a head's largest bias to its running maximum: weights must not underflow


@dataclass(frozen=True)
class Difference:
    """How the two maps of a head are combined."""

    weight: float  # lambda
    scale: float
    eps: float
    dim: int  # real value channels


@dataclass(frozen=True)
class ValueTurn:
    """Values divided by their root mean square over ``dim`` channels and rotated by their position before they are cached."""

    rope: torch.Tensor  # [positions, dim / 2, 2]
    dim: int


@dataclass
class DistanceBias:
    """Per head, what a key ``n`` tokens back adds to its score: ``table[h, min(n, last)]``."""

    table: torch.Tensor  # [heads, last + 1] fp32
    top: torch.Tensor  # [heads] largest entry

    @classmethod
    def from_table(cls, table: torch.Tensor) -> "DistanceBias":
        table = table.float().contiguous()
        if float((table.amax(1) - table.amin(1)).max()) > MAX_BIAS_SPREAD:
            raise ValueError(f"biases of a head that differ by more than {MAX_BIAS_SPREAD:g} are not supported")
        return cls(table, table.amax(1).contiguous())

    @property
    def last(self) -> int:
        return self.table.shape[1] - 1


def log_buckets(rows: int, most: float) -> list[int]:
    """Row of a table of ``rows`` for the distances 0, 1, ...: one row each up to half of them, then logarithmic up to ``most``; ends
    where the last row begins."""
    half, out = rows // 2, []
    while not out or out[-1] < rows - 1:
        n = len(out)
        out.append(n if n < half else min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half))))
    return out


@dataclass(frozen=True)
class LinearScaling:
    """Every rotation frequency divided by ``factor``."""

    factor: float

    def __call__(self, f: float) -> float:
        return f / self.factor


@dataclass(frozen=True)
class FrequencyScaling:
    """Rotation frequencies for contexts longer than the original one: frequencies that turn less than ``low`` times over the
    original context are divided by ``factor``, those that turn more than ``high`` times are kept, with a linear blend between."""

    factor: float
    low: float
    high: float
    original: float

    def __call__(self, f: float) -> float:
        turns = self.original * f / (2 * math.pi)
        if turns > self.high:
            return f
        if turns < self.low:
            return f / self.factor
        s = (turns - self.low) / (self.high - self.low) if self.high > self.low else 1.0
        return (1 - s) * f / self.factor + s * f


def rope_table(base: float, dims: int, positions: int, device, scaling=None) -> torch.Tensor:
    """``[positions, dims / 2, 2]`` fp32 (cos, sin) of ``p * f_i``, ``f_i = base^(-2i / dims)``, in double precision.  ``scaling``: a
    :class:`FrequencyScaling`, a :class:`LinearScaling`, or a :class:`~mfq_b200.models.rope_scaling.YarnScaling`, which also lengthens the rotated pairs."""
    freq, length = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], 1.0
    if isinstance(scaling, (FrequencyScaling, LinearScaling)):
        freq = [scaling(f) for f in freq]
    elif scaling is not None:
        freq, length = scaling.frequencies(dims, base), scaling.mscale
    a = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * torch.tensor(freq, dtype=torch.float64, device=device)
    return (torch.stack([a.cos(), a.sin()], -1) * length).float().contiguous()


def qkv_finish(qkv: torch.Tensor, kv, positions, slots, *, heads: int, kv_heads: int, dim: int, q_norm, k_norm, rope, rot: int,
               eps: float, v_first: torch.Tensor | None = None, mix: float = 0.0, maps: int = 1, pairs: bool = False,
               dk: int | None = None, temperature: tuple[float, int] | None = None, turn: ValueTurn | None = None) -> torch.Tensor:
    """Per-head RMS norm of q and k (over ``dim`` channels; no norm without weights), rotation of the leading ``rot`` channels
    (``i`` with ``i + rot / 2``, or with its neighbour: ``pairs``), K and V into their pages; returns ``q [T, maps * heads, dk]``.
    ``v_first`` (``[T, kv_heads * dv]``, rows may be strided): the cached values are ``(1 - mix) v + mix v_first``.  ``kv`` None:
    the rows hold queries only (of stored width ``dk``).  ``temperature`` (coef, every): queries at position p times
    ``1 + coef * ln(floor((p + 1) / every) + 1)``.  ``turn``: values are normed and rotated, in the same layout of pairs."""
    t = qkv.shape[0]
    if kv is not None:
        dk, dv, page = kv.k.shape[-1] // maps, kv.v.shape[-1], kv.page_size
    else:
        dv = page = 0
    q = torch.empty((t, maps * heads, dk), dtype=qkv.dtype, device=qkv.device)
    temp, every = temperature or (0.0, 1)
    rc = dense_lib().mfq_qkv_finish(ptr(qkv), qkv.stride(0), ptr(v_first), v_first.stride(0) if v_first is not None else 0, float(mix),
                                    ptr(q), ptr(kv.k) if kv is not None else None, ptr(kv.v) if kv is not None else None, ptr(positions),
                                    ptr(slots), ptr(q_norm), ptr(k_norm), ptr(rope), rope.shape[0] if rope is not None else 0, t,
                                    maps * heads, kv_heads, maps, dim, dk, dv, rot, int(pairs), page, float(eps), float(temp), int(every), ptr(turn.rope) if turn is not None else None,
                                    turn.dim if turn is not None else 0, turn.rope.shape[0] if turn is not None else 0, is_fp32(qkv.dtype), stream_ptr())
    check(rc, "qkv_finish")
    return q


def difference(a: torch.Tensor, kv_heads: int, d: Difference, out: torch.Tensor | None = None) -> torch.Tensor:
    """``a [T, 2 * H, dv]`` (both maps of every head, in query order) -> ``[T, H, dv]``."""
    t, rows, dv = a.shape
    out = torch.empty((t, rows // 2, dv), dtype=a.dtype, device=a.device) if out is None else out
    check(dense_lib().mfq_map_difference(ptr(a), ptr(out), t, rows // 2, rows // 2 // kv_heads, dv, d.dim, d.weight, d.scale, d.eps,
                                         is_fp32(a.dtype), stream_ptr()), "map_difference")
    return out


def turn_back(o: torch.Tensor, turn: ValueTurn, positions, pairs: bool = False) -> torch.Tensor:
    """``o [T, H, dv]`` in place: every head's output turned by minus the token's position."""
    t, h, dv = o.shape
    check(dense_lib().mfq_turn_back(ptr(o), ptr(turn.rope), ptr(positions), t, h, dv, turn.dim, turn.rope.shape[0], int(pairs), is_fp32(o.dtype),
                                    stream_ptr()), "turn_back")
    return o


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


def _bias_args(bias: DistanceBias | None) -> tuple:
    return (ptr(bias.table), bias.last) if bias is not None else (None, 0)


def decode(q: torch.Tensor, kv, block_table, seq_lens, *, window: int, scale: float, cap: float, keep: int = 0,
           diff: Difference | None = None, bias: DistanceBias | None = None, sink: torch.Tensor | None = None, chunk: int = 0,
           turn: ValueTurn | None = None, splits: int = 1, out=None):
    """One query token per sequence (bf16): ``q [B, Hq, dk]`` -> ``[B, Hq, dv]``, or ``[B, Hq / 2, dv]`` with ``diff``;
    ``seq_lens`` count the query token.  ``turn``: outputs turn back (halves; one map)."""
    b, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    maps = 1 if diff is None else 2
    out = torch.empty((b, hq // maps, dv), dtype=q.dtype, device=q.device) if out is None else out
    ws = Workspace.get(q.device)
    parts = splits > 1 or maps > 1
    assert kv.k.shape[-1] == maps * dk
    assert not parts or (b * hq * splits * dv <= ws.attn_acc.numel() and b * hq * splits * 2 <= ws.attn_ml.numel())
    how = (diff.weight, diff.scale, diff.eps, diff.dim) if diff is not None else (0.0, 1.0, 0.0, dv)
    rc = dense_lib().mfq_window_attn_decode(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(seq_lens), ptr(out), ptr(ws.attn_acc),
                                            ptr(ws.attn_ml), b, hq, hk, maps, dk, dv, block_table.stride(0), window, chunk, keep, float(scale),
                                            float(cap), splits, *how, *_bias_args(bias), ptr(sink), ptr(turn.rope) if turn is not None else None,
                                            turn.dim if turn is not None else 0, turn.rope.shape[0] if turn is not None else 0, stream_ptr())
    check(rc, "window_attn_decode", 2 if parts else 1)
    return out


def prefill(q: torch.Tensor, kv, block_table, q_starts, seq_lens, max_q: int, *, window: int, scale: float, cap: float, keep: int = 0,
            maps: int = 1, bias: DistanceBias | None = None, sink: torch.Tensor | None = None, chunk: int = 0, out=None):
    """Portions of several sequences (bf16): rows ``q_starts[b] .. q_starts[b + 1] - 1`` of ``q [T, Hq, dk]`` are the last
    tokens of a sequence of ``seq_lens[b]``.  ``max_q``: the longest portion (host).  Writes the output of every map."""
    t, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    out = torch.empty((t, hq, dv), dtype=q.dtype, device=q.device) if out is None else out
    rc = dense_lib().mfq_window_attn_prefill(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(q_starts), ptr(seq_lens), ptr(out), t,
                                             seq_lens.numel(), max_q, hq, hk, maps, dk, dv, kv.k.shape[0], block_table.stride(0), window, chunk,
                                             keep, float(scale), float(cap), *_bias_args(bias), ptr(bias.top) if bias is not None else None, ptr(sink),
                                             ptr(Workspace.get(q.device).status), stream_ptr())
    check(rc, "window_attn_prefill")
    return out


def plain(q: torch.Tensor, kv, block_table, tok_seq, positions, *, window: int, scale: float, cap: float, keep: int = 0, maps: int = 1,
          bias: DistanceBias | None = None, sink: torch.Tensor | None = None, chunk: int = 0):
    """The same in fp32 arithmetic for any mix of tokens: token ``t`` is at ``positions[t]`` of sequence ``tok_seq[t]``."""
    t, hq, dk = q.shape
    hk, dv = kv.k.shape[1], kv.v.shape[-1]
    out = torch.empty((t, hq, dv), dtype=q.dtype, device=q.device)
    rc = dense_lib().mfq_window_attn_plain(ptr(q), ptr(kv.k), ptr(kv.v), ptr(block_table), ptr(tok_seq), ptr(positions), ptr(out), t, hq,
                                           hk, maps, dk, dv, block_table.stride(0), window, chunk, keep, float(scale), float(cap),
                                           *_bias_args(bias), ptr(sink), is_fp32(q.dtype), stream_ptr())
    check(rc, "window_attn_plain")
    return out


def visible_keys(length: int, window: int, keep: int) -> int:
    """Most keys a query of a sequence of ``length`` tokens sees."""
    return min(length, window + keep)

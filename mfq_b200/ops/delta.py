"""Delta rule with a decay per key channel (``csrc/delta.cu``, ``csrc/delta_chunk.cu``) and the short convolution in front of it
(``csrc/mix_ops.cu``).

Per value head (key head ``h / (H / G)``), with a fp32 state ``S [dk, dv]`` carried from token to token and unit vectors ``q`` (also
times ``dim^-1/2``) and ``k``:

    g_t = exp(-exp(A_log) softplus(W_a2 a_t + dt_bias));   beta_t = sigmoid(b_t)
    S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
    y_t = rms(o_t) * norm_w * sigmoid(W_g2 g1_t)

A token's projections are one row ``[q: G dk | k: G dk | v: H dv | b: up(H) | a: ra | g1: rg]``; the first three pass a causal
convolution over time and SiLU.  bf16 portions of prompts run in 64-token chunks, single tokens, short portions and fp32 token by token.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .dense import DenseLinear, is_fp32, up
from .lib import Workspace, check, dense_lib, ptr, stream_ptr

CHUNK, CHUNK_MAX_DK, CHUNK_MAX_RANK = 64, 128, 64
CHUNKED_MIN_TOKENS = 16  # a batch whose longest portion is shorter goes token by token
_scratch: dict[int, torch.Tensor] = {}
MAX_ROWS, THREADS, MAX_SPLIT = 16, 256, 8  # of the token-by-token kernel


@dataclass(frozen=True)
class Geometry:
    heads: int
    key_heads: int
    dk: int  # as stored
    dv: int
    dim: int  # real widths
    vdim: int
    rank_a: int  # as stored
    rank_g: int
    taps: int
    eps: float

    @property
    def channels(self) -> int:
        """Columns that pass the convolution."""
        return 2 * self.key_heads * self.dk + self.heads * self.dv

    @property
    def b_cols(self) -> int:
        return up(self.heads)

    @property
    def width(self) -> int:
        """Columns of a row of projections."""
        return self.channels + self.b_cols + self.rank_a + self.rank_g

    @property
    def chunkable(self) -> bool:
        return self.dk <= CHUNK_MAX_DK and self.dv <= 1024 and self.rank_a <= CHUNK_MAX_RANK and self.rank_a % 16 == 0

    def chunk_bytes(self) -> int:
        """Scratch per chunk and head."""
        rows = CHUNK * (self.dk + 8) * 2
        return 6 * rows + 2 * CHUNK * 72 * 2 + 4 * self.dk + CHUNK * self.dv * 4


@dataclass
class Weights:
    conv: torch.Tensor  # [taps, channels] fp32, last row for the current token
    a2: torch.Tensor  # [H * dk, ra]
    dt_bias: torch.Tensor  # [H * dk] fp32
    rate: torch.Tensor  # [H] fp32, exp(A_log)
    g2: DenseLinear  # [H * dv, rg]
    norm: torch.Tensor  # [dv] fp32


def column_split(batch: int, heads: int, dk: int, dv: int) -> int:
    """CTAs over a head's value columns: as many as the kernel's registers need, more while the grid leaves SMs free; 0: the sizes do
    not fit."""
    fits = lambda s: dv % (4 * s) == 0 and dv // s // 4 <= THREADS and -(-dk // min(dk, THREADS // (dv // s // 4))) <= MAX_ROWS
    s = next((s for s in range(1, MAX_SPLIT + 1) if fits(s)), 0)
    while s and s * 2 <= MAX_SPLIT and batch * heads * s * 2 <= 148 and fits(s * 2) and dv // (s * 2) >= 16:
        s *= 2
    return s


def conv(proj: torch.Tensor, w: torch.Tensor, state: torch.Tensor, slots: torch.Tensor, channels: int, *, starts: torch.Tensor | None = None,
         max_q: int = 1, bias: torch.Tensor | None = None, out: torch.Tensor | None = None) -> torch.Tensor:
    """``silu(causal convolution (+ bias))`` of the first ``channels`` columns; ``state [slots, taps - 1, channels]`` keeps the last inputs;
    ``starts [B + 1]``: first row of every portion, or None for one row per sequence."""
    out = torch.empty((proj.shape[0], channels), dtype=proj.dtype, device=proj.device) if out is None else out
    rc = dense_lib().mfq_short_conv(ptr(proj), proj.stride(0), ptr(w), ptr(bias), ptr(state), ptr(slots), ptr(starts), ptr(out), out.stride(0), slots.numel(),
                                    max_q, channels, w.shape[0], is_fp32(proj.dtype), stream_ptr())
    check(rc, "short_conv", 2 if starts is not None and w.shape[0] > 1 else 1)
    return out


def recurrent(x: torch.Tensor, proj: torch.Tensor, w: Weights, state: torch.Tensor, slots: torch.Tensor, geo: Geometry, *,
              starts: torch.Tensor | None = None, out: torch.Tensor | None = None, split: int | None = None) -> torch.Tensor:
    """Token by token.  ``x [T, channels]`` behind the convolution, ``proj [T, width]``, ``state [slots, H, dk, dv]``, ``slots [B]``
    (< 0: the sequence is skipped).  Returns ``y [T, H * dv]``."""
    b = slots.numel()
    out = torch.empty((x.shape[0], geo.heads * geo.dv), dtype=x.dtype, device=x.device) if out is None else out
    split = column_split(b, geo.heads, geo.dk, geo.dv) if split is None else split
    side = proj[:, geo.channels :]
    rc = dense_lib().mfq_delta_recurrent(ptr(x), ptr(side), ptr(w.a2), ptr(w.g2.w), ptr(w.dt_bias), ptr(w.rate), ptr(w.norm), ptr(out), ptr(state),
                                         ptr(slots), ptr(starts), b, geo.heads, geo.key_heads, geo.dk, geo.dv, geo.vdim, geo.b_cols,
                                         geo.rank_a, geo.rank_g, x.stride(0), proj.stride(0), split, geo.dim ** -0.5, geo.eps,
                                         is_fp32(x.dtype), stream_ptr())
    check(rc, "delta_recurrent")
    return out


def chunked(x: torch.Tensor, proj: torch.Tensor, w: Weights, state: torch.Tensor, slots: torch.Tensor, geo: Geometry, starts: torch.Tensor,
            max_q: int, *, first: int = 0, out: torch.Tensor | None = None) -> torch.Tensor:
    """The same for portions (bf16), 64 tokens at a time; ``max_q``: the longest portion, ``first``: the first row of any (host)."""
    t, b, dev = x.shape[0], slots.numel(), x.device.index or 0
    out = torch.empty((t, geo.heads * geo.dv), dtype=x.dtype, device=x.device) if out is None else out
    chunks = (t - first) // CHUNK + b
    need = chunks * geo.heads * geo.chunk_bytes()
    if dev not in _scratch or _scratch[dev].numel() < need:
        _scratch[dev] = torch.empty(need, dtype=torch.uint8, device=x.device)
    side = proj[:, geo.channels :]
    gate = w.g2(side[:, geo.b_cols + geo.rank_a :])
    raw = torch.empty((t, geo.heads * geo.dv), dtype=torch.float32, device=x.device)
    rc = dense_lib().mfq_delta_chunk(ptr(x), ptr(side), ptr(w.a2), ptr(gate), ptr(w.dt_bias), ptr(w.rate), ptr(w.norm), ptr(out), ptr(state),
                                     ptr(slots), ptr(starts), ptr(raw), ptr(_scratch[dev]), chunks, first, t - first, b, max_q, geo.heads,
                                     geo.key_heads, geo.dk, geo.dv, geo.vdim, geo.b_cols, geo.rank_a, geo.rank_g, x.stride(0), proj.stride(0),
                                     geo.dim ** -0.5, geo.eps, ptr(Workspace.get(x.device).status), stream_ptr())
    check(rc, "delta_chunk", 3)
    return out


def ragged(proj: torch.Tensor, w: Weights, state: torch.Tensor, conv_state: torch.Tensor, slots: torch.Tensor, geo: Geometry,
           starts: torch.Tensor | None, max_q: int, singles: int) -> torch.Tensor:
    """Convolution and recurrence of a batch of portions whose first ``singles`` sequences bring one token each (``starts`` None: all)."""
    x = torch.empty((proj.shape[0], geo.channels), dtype=proj.dtype, device=proj.device)
    out = torch.empty((proj.shape[0], geo.heads * geo.dv), dtype=proj.dtype, device=proj.device)
    singles = slots.numel() if starts is None else singles
    if singles:
        conv(proj, w.conv, conv_state, slots[:singles], geo.channels, out=x)
        recurrent(x, proj, w, state, slots[:singles], geo, out=out)
    if singles < slots.numel():
        rest, first = slots[singles:], starts[singles:]
        conv(proj, w.conv, conv_state, rest, geo.channels, starts=first, max_q=max_q, out=x)
        if proj.dtype == torch.bfloat16 and max_q >= CHUNKED_MIN_TOKENS and geo.chunkable:
            chunked(x, proj, w, state, rest, geo, first, max_q, first=singles, out=out)
        else:
            recurrent(x, proj, w, state, rest, geo, starts=first, out=out)
    return out

"""Gated linear attention (``csrc/gla.cu``, ``csrc/gla_chunk.cu``).

Per head, with a fp32 state ``S [dk, dv]`` carried from token to token:

    alpha_t = sigmoid(W_a2 a_t + bias)^(1 / tau);   S <- diag(alpha_t) S + k_t v_t^T;   o_t = S^T (q_t scale)
    y_t = rms(o_t) * norm_w * silu(gate_t)

or, with a bonus ``u`` (time mixing), ``o_t = (S + diag(u) k_t v_t^T)^T (q_t scale)`` from the state before the write.  The decay may
instead be ``exp(-exp(W_a2 a_t + bias))``, and every head may have norm weights of its own.

A token's projections are one row ``[q: H dk | k: H dk | v: H dv | gate: H dv | a: rank]`` (widths and the
rank stored as multiples of 16).  bf16 portions of prompts run in 64-token chunks, single tokens, short portions and fp32 token by token.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .dense import is_fp32
from .lib import check, dense_lib, ptr, stream_ptr

CHUNK = 64
CHUNKED_MIN_TOKENS = 16  # a batch whose longest portion is shorter goes token by token
_scratch: dict[tuple[int, str], torch.Tensor] = {}


@dataclass(frozen=True)
class Geometry:
    heads: int
    dk: int  # as stored
    dv: int
    dim: int  # real widths
    vdim: int
    rank: int  # as stored
    tau: float
    eps: float
    decay: str = "sigmoid"  # or "exp": exp(-exp(z))
    scaled: bool = True  # whether q is multiplied by dim^-1/2

    @property
    def scale(self) -> float:
        return self.dim ** -0.5 if self.scaled else 1.0

    def shape_args(self, norm_w, bonus) -> tuple:
        """How z becomes a decay, the stride of the norm weights, the bonus."""
        assert norm_w.numel() in (self.dv, self.heads * self.dv)
        return ("sigmoid", "exp").index(self.decay), self.dv if norm_w.dim() == 2 else 0, ptr(bonus)

    @property
    def width(self) -> int:
        """Columns of a row of projections."""
        return 2 * self.heads * (self.dk + self.dv) + self.rank

    @property
    def chunkable(self) -> bool:
        return self.dk <= 256 and self.dv <= 512 and self.rank <= 64 and self.rank % 16 == 0


def _space(name: str, floats: int, device) -> torch.Tensor:
    key = (device.index or 0, name)
    t = _scratch.get(key)
    if t is None or t.numel() < floats:
        t = _scratch[key] = torch.empty(floats, dtype=torch.float32, device=device)
    return t


def _split(batch: int, heads: int, dv: int) -> int:
    """CTAs over a head's value columns: only while the grid leaves SMs free."""
    s = 1
    while s < 8 and batch * heads * s * 2 <= 148 and dv % (8 * s) == 0 and dv // (s * 2) >= 16:
        s *= 2
    return s


def recurrent(proj: torch.Tensor, w2, bias, norm_w, state, slots, geo: Geometry, *, starts: torch.Tensor | None = None,
              out: torch.Tensor | None = None, split: int | None = None, bonus: torch.Tensor | None = None) -> torch.Tensor:
    """Token by token.  ``norm_w [dv]`` or ``[H, dv]``; ``bonus [H * dk]``.  ``proj [T, width]``, ``state [slots, H, dk, dv]``, ``slots [B]`` (< 0: the sequence is skipped);
    ``starts [B + 1]``: first row of every portion, or None for one row per sequence.  Returns ``y [T, H * dv]``."""
    b = slots.numel()
    out = torch.empty((proj.shape[0], geo.heads * geo.dv), dtype=proj.dtype, device=proj.device) if out is None else out
    split = _split(b, geo.heads, geo.dv) if split is None else split
    rc = dense_lib().mfq_gla_recurrent(ptr(proj), ptr(w2), ptr(bias), ptr(norm_w), ptr(out), ptr(state), ptr(slots), ptr(starts), b,
                                       geo.heads, geo.dk, geo.dv, geo.vdim, geo.rank, proj.stride(0), split, geo.scale, 1.0 / geo.tau,
                                       geo.eps, *geo.shape_args(norm_w, bonus), is_fp32(proj.dtype), stream_ptr())
    check(rc, "gla_recurrent")
    return out


def chunked(proj: torch.Tensor, w2, bias, norm_w, state, slots, geo: Geometry, starts: torch.Tensor, max_q: int,
            out: torch.Tensor | None = None, bonus: torch.Tensor | None = None) -> torch.Tensor:
    """The same for portions (bf16), 64 tokens at a time; ``max_q``: the longest portion (host)."""
    t, b = proj.shape[0], slots.numel()
    out = torch.empty((t, geo.heads * geo.dv), dtype=proj.dtype, device=proj.device) if out is None else out
    chunks, keys = t // CHUNK + b, geo.heads * geo.dk
    cum, u = _space("cum", t * keys, proj.device), _space("u", chunks * keys * geo.dv, proj.device)
    gam = _space("gam", chunks * keys, proj.device)
    rc = dense_lib().mfq_gla_chunk(ptr(proj), ptr(w2), ptr(bias), ptr(norm_w), ptr(out), ptr(state), ptr(slots), ptr(starts), ptr(cum),
                                   ptr(u), ptr(gam), b, max_q, geo.heads, geo.dk, geo.dv, geo.vdim, geo.rank, proj.stride(0),
                                   geo.scale, 1.0 / geo.tau, geo.eps, *geo.shape_args(norm_w, bonus), stream_ptr())
    check(rc, "gla_chunk", 3)
    return out


def ragged(proj: torch.Tensor, w2, bias, norm_w, state, slots, geo: Geometry, starts: torch.Tensor, max_q: int, singles: int,
           bonus: torch.Tensor | None = None) -> torch.Tensor:
    """A batch of portions whose first ``singles`` sequences bring one token each."""
    out = torch.empty((proj.shape[0], geo.heads * geo.dv), dtype=proj.dtype, device=proj.device)
    if singles:
        recurrent(proj, w2, bias, norm_w, state, slots[:singles], geo, out=out, bonus=bonus)
    if singles < slots.numel():
        if proj.dtype == torch.bfloat16 and max_q >= CHUNKED_MIN_TOKENS and geo.chunkable:
            chunked(proj, w2, bias, norm_w, state, slots[singles:], geo, starts[singles:], max_q, out=out, bonus=bonus)
        else:
            recurrent(proj, w2, bias, norm_w, state, slots[singles:], geo, starts=starts[singles:], out=out, bonus=bonus)
    return out


def token_shift(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, slots, starts: torch.Tensor | None = None,
                tok_seq: torch.Tensor | None = None) -> torch.Tensor:
    """``[T, streams * W]``: stream s of a token reads ``h + (h' - h) * mu[s]``, ``h'`` the previous token's row of ``h [T, W]``.
    ``last [slots, W]`` fp32 keeps every sequence's last row (zeros before its first); ``starts`` None: one row per sequence."""
    t, w = h.shape
    out = torch.empty((t, mu.shape[0] * w), dtype=h.dtype, device=h.device)
    check(dense_lib().mfq_token_shift(ptr(h), ptr(mu), ptr(last), ptr(slots), ptr(starts), ptr(tok_seq), ptr(out), t, w, mu.shape[0],
                                      is_fp32(h.dtype), stream_ptr()), "token_shift")
    return out

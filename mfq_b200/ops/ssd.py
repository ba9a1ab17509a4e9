"""State-space recurrence with one decay per head (``csrc/ssd.cu``, ``csrc/ssd_chunk.cu``), its short convolution
(:func:`~mfq_b200.ops.delta.conv`) and the gated norm behind it.

Per head (of group ``h / (H / groups)``), with a fp32 state ``S [N, P]`` carried from token to token:

    dt_t = softplus(z_t + dt_bias);   S <- exp(-rate dt_t) S + dt_t B_t x_t^T;   y_t = S^T C_t + skip x_t
    out  = rms(y silu(z)) * norm_w, the root mean square over each of ``parts`` equal runs of channels

A token's projections are one row ``[x: H P | B: groups N | C: groups N | z: H P | dt: up(H)]``; the first three pass a causal
convolution over time and SiLU.  bf16 portions of prompts run in chunks, single tokens, short portions and fp32 token by token.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .delta import conv
from .dense import is_fp32, up
from .lib import check, dense_lib, ptr, stream_ptr

CHUNKED_MIN_TOKENS = 16  # a batch whose longest portion is shorter goes token by token
CHUNK_SMEM, THREADS, MAX_ROWS = 227 * 1024, 256, 16
_scratch: dict[int, torch.Tensor] = {}


@dataclass(frozen=True)
class Geometry:
    heads: int
    groups: int
    state: int  # as stored (N)
    width: int  # as stored (P)
    vdim: int  # real channels of a head
    taps: int
    parts: int
    eps: float

    @property
    def inner(self) -> int:
        return self.heads * self.width

    @property
    def channels(self) -> int:
        """Columns that pass the convolution."""
        return self.inner + 2 * self.groups * self.state

    @property
    def row(self) -> int:
        """Columns of a row of projections."""
        return self.channels + self.inner + up(self.heads)

    def chunk_fits(self, chunk: int, heads: int = 1) -> bool:
        """Whether a chunk of this many tokens fits the shared memory of its kernels."""
        return 2 * chunk * (self.state + 8) * 2 + chunk * 144 + self.state * 272 + 8 * heads * chunk <= CHUNK_SMEM


@dataclass
class Weights:
    conv: torch.Tensor  # [taps, channels] fp32, last row for the current token
    conv_bias: torch.Tensor  # [channels] fp32
    dt_bias: torch.Tensor  # [H] fp32
    rate: torch.Tensor  # [H] fp32, exp(A_log)
    skip: torch.Tensor  # [H] fp32
    norm: torch.Tensor  # [H * P] fp32, zero in padding channels


def column_split(batch: int, heads: int, n: int, p: int) -> int:
    """CTAs over a head's columns: as many as the kernel's registers need, more while the grid leaves SMs free; 0: the sizes do not
    fit."""
    def fits(s):
        if p % (4 * s) or p // s // 4 > THREADS:
            return False
        return -(-n // min(n, THREADS // (p // s // 4))) <= MAX_ROWS
    s = next((s for s in range(1, 17) if fits(s)), 0)
    while s and batch * heads * s * 2 <= 148 and fits(s * 2) and p // (s * 2) >= 16:
        s *= 2
    return s


def _args(x: torch.Tensor, proj: torch.Tensor, w: Weights, geo: Geometry, out: torch.Tensor, state: torch.Tensor, slots, starts) -> tuple:
    dt = proj[:, geo.channels + geo.inner :]
    return (ptr(x), ptr(dt), ptr(w.dt_bias), ptr(w.rate), ptr(w.skip), ptr(out), ptr(state), ptr(slots), ptr(starts))


def recurrent(x: torch.Tensor, proj: torch.Tensor, w: Weights, state: torch.Tensor, slots: torch.Tensor, geo: Geometry, *,
              starts: torch.Tensor | None = None, out: torch.Tensor | None = None, split: int | None = None) -> torch.Tensor:
    """Token by token.  ``x [T, channels]`` behind the convolution, ``proj [T, row]``, ``state [slots, H, N, P]``, ``slots [B]`` (< 0: the
    sequence is skipped); ``starts [B + 1]``: first row of every portion, or None for one row per sequence.  Returns ``y [T, H * P]``."""
    b = slots.numel()
    out = torch.empty((x.shape[0], geo.inner), dtype=x.dtype, device=x.device) if out is None else out
    split = column_split(b, geo.heads, geo.state, geo.width) if split is None else split
    check(dense_lib().mfq_ssd_recurrent(*_args(x, proj, w, geo, out, state, slots, starts), b, geo.heads, geo.groups, geo.state, geo.width,
                                        x.stride(0), proj.stride(0), split, is_fp32(x.dtype), stream_ptr()), "ssd_recurrent")
    return out


def chunk_plan(geo: Geometry, tokens: int, longest: int) -> tuple[int, int]:
    """``(tokens of a chunk, heads of a CTA)``: more heads share the scores of their group as long as the grid stays large."""
    chunk = 128 if longest > 64 and geo.chunk_fits(128) else 64
    heads, per = 1, geo.heads // geo.groups
    while per % (2 * heads) == 0 and heads < 8 and -(-tokens // chunk) * geo.heads // (2 * heads) >= 3 * 148 and geo.chunk_fits(chunk, 2 * heads):
        heads *= 2
    return chunk, heads


def chunked(x: torch.Tensor, proj: torch.Tensor, w: Weights, state: torch.Tensor, slots: torch.Tensor, geo: Geometry, starts: torch.Tensor,
            max_q: int, *, first: int = 0, out: torch.Tensor | None = None, chunk: int | None = None, heads: int | None = None) -> torch.Tensor:
    """The same for portions (bf16), 64 or 128 tokens at a time; ``max_q``: the longest portion, ``first``: the first row of any (host)."""
    t, b, dev = x.shape[0] - first, slots.numel(), x.device.index or 0
    out = torch.empty((x.shape[0], geo.inner), dtype=x.dtype, device=x.device) if out is None else out
    plan = chunk_plan(geo, t, max_q)
    chunk, heads = (plan[0] if chunk is None else chunk), (plan[1] if heads is None else heads)
    chunks = t // chunk + b
    states = chunks * geo.heads * geo.state * geo.width
    need = states + chunks * geo.heads
    if dev not in _scratch or _scratch[dev].numel() < need:
        _scratch[dev] = torch.empty(need, dtype=torch.float32, device=x.device)
    u, gam = _scratch[dev], _scratch[dev][states:]
    check(dense_lib().mfq_ssd_chunk(*_args(x, proj, w, geo, out, state, slots, starts), ptr(u), ptr(gam), b, max_q, geo.heads, geo.groups, geo.state,
                                    geo.width, x.stride(0), proj.stride(0), chunk, heads, stream_ptr()), "ssd_chunk", 3)
    return out


def gate_norm(y: torch.Tensor, proj: torch.Tensor, w: Weights, geo: Geometry) -> torch.Tensor:
    """``rms(y silu(z)) * norm`` in :attr:`Geometry.parts` runs of the real channels."""
    out, z = torch.empty_like(y), proj[:, geo.channels :]
    check(dense_lib().mfq_ssd_gate_norm(ptr(y), ptr(z), ptr(w.norm), ptr(out), y.shape[0], geo.heads, geo.width, geo.vdim, proj.stride(0), geo.parts,
                                        float(geo.eps), is_fp32(y.dtype), stream_ptr()), "ssd_gate_norm")
    return out


def ragged(proj: torch.Tensor, w: Weights, state: torch.Tensor, conv_state: torch.Tensor, slots: torch.Tensor, geo: Geometry,
           starts: torch.Tensor | None, max_q: int, singles: int) -> torch.Tensor:
    """Convolution, recurrence and gated norm of a batch of portions whose first ``singles`` sequences bring one token each (``starts``
    None: all)."""
    x = torch.empty((proj.shape[0], geo.channels), dtype=proj.dtype, device=proj.device)
    y = torch.empty((proj.shape[0], geo.inner), dtype=proj.dtype, device=proj.device)
    singles = slots.numel() if starts is None else singles
    if singles:
        conv(proj, w.conv, conv_state, slots[:singles], geo.channels, bias=w.conv_bias, out=x)
        recurrent(x, proj, w, state, slots[:singles], geo, out=y)
    if singles < slots.numel():
        rest, first = slots[singles:], starts[singles:]
        conv(proj, w.conv, conv_state, rest, geo.channels, starts=first, max_q=max_q, bias=w.conv_bias, out=x)
        if proj.dtype == torch.bfloat16 and max_q >= CHUNKED_MIN_TOKENS and geo.chunk_fits(64):
            chunked(x, proj, w, state, rest, geo, first, max_q, first=singles, out=y)
        else:
            recurrent(x, proj, w, state, rest, geo, starts=first, out=y)
    return gate_norm(y, proj, w, geo)

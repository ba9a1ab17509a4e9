"""Unquantized linears and the fp32 residual stream (``csrc/dense_gemm.cu``, ``csrc/stream_ops.cu``).

Activations and weights are bf16, or fp32 throughout; the element type of the weight decides.  Stored widths are rounded up
(:func:`up`) and the padding is zero, so the kernels need no tails; callers keep the true widths where they matter (norms).
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .lib import Workspace, check, dense_lib, ptr, stream_ptr

BIAS, GLU, GELU, GELU_GLU, SOFTCAP, ADD, RELU_GLU, SILU_GLU, FLOAT, RELU2 = range(10)  # epilogues (dense_common.cuh)
UNITS = {"gelu": GELU_GLU, "relu": RELU_GLU, "silu": SILU_GLU}  # act(gate) * up
ACTIVATIONS = {"relu2": RELU2}  # max(y, 0)^2
GEMV_ROWS, GEMV_MID_ROWS, GEMV_MID_WEIGHTS = 8, 16, 8 << 20


def up(n: int, m: int = 16) -> int:
    """``n`` rounded up to a multiple of ``m``."""
    return (n + m - 1) // m * m


def is_fp32(dtype: torch.dtype) -> int:
    if dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"the dense path runs in bfloat16 or float32, not {dtype}")
    return int(dtype == torch.float32)


def _most_splits(tiles: int, blocks: int, small: bool, sms: int) -> int:
    """Most K splits worth taking: the clusters must all be resident at once, every CTA keeps 8 K blocks.  Where one CTA fills
    an SM, clusters do not pack every SM of a GPC: 128 CTAs fit, 96 in clusters of more than 4."""
    best = 1
    for s in range(2, 9):
        room = sms if small else (96 if s > 4 else 128)
        if tiles * s <= room and blocks // s >= 8:
            best = s
    return best


def plan(m: int, n: int, k: int, sms: int = 148) -> tuple[int, int]:
    """``(token tile, K splits)`` of a bf16 product ``[m, k] x [n, k]^T``; tile 0 is the weight-streaming kernel.  Fitted to a
    sweep on B200 over the projections of 1B- and 8B-sized layers at 16 .. 4096 tokens: up to 128 tokens the weights are read
    once whatever the split, so the grid is filled; beyond that a wave of 256-token tiles costs about 7 + 0.35 us per K block,
    of 128-token tiles 5 + 0.30 us, and meeting in a cluster 5 / 3 us."""
    if m <= GEMV_ROWS or (m <= GEMV_MID_ROWS and n * k <= GEMV_MID_WEIGHTS):
        return 0, 1
    rows, blocks = math.ceil(n / 128), math.ceil(k / 64)
    for tile in (16, 32, 64, 128):
        if m <= tile:
            return tile, _most_splits(rows, blocks, tile <= 64, sms)
    best, best_cost = (128, 1), None
    for tile, ramp, per_block, meet in ((128, 5.0, 0.30, 3.0), (256, 7.0, 0.35, 5.0)):
        tiles = rows * math.ceil(m / tile)
        for s in range(1, _most_splits(tiles, blocks, False, sms) + 1):
            cost = math.ceil(tiles * s / sms) * (ramp + per_block * math.ceil(blocks / s)) + (meet if s > 1 else 0.0)
            if best_cost is None or cost < best_cost:
                best, best_cost = (tile, s), cost
    return best


@dataclass
class DenseLinear:
    """``[rows, cols]`` weight (rows a multiple of 16, cols of 8) with an optional fp32 bias.  ``glu``: the rows alternate
    between 8 gate and 8 up rows (:func:`interleave_glu`) and the output is the gated unit of the two, half as wide.
    ``act``: an activation of the output without a gate (:data:`ACTIVATIONS`).  ``groups`` G > 1: G matrices on top of each other,
    ``[G * rows, cols]``, each with its own columns of input and output."""

    w: torch.Tensor
    bias: torch.Tensor | None = None
    glu: tuple[float, float] | str | None = None  # (alpha, limit) of the clipped GLU, or the activation: act(gate) * up
    groups: int = 1
    act: str | None = None
    input_kind = "dense"

    @property
    def out_width(self) -> int:
        return self.w.shape[0] // self.groups // (2 if self.glu is not None else 1)

    def __call__(self, x: torch.Tensor, *, table: torch.Tensor | None = None, ids: torch.Tensor | None = None,
                 softcap: float = 0.0, add_to: torch.Tensor | None = None, scale: float = 1.0, out: torch.Tensor | None = None,
                 fp32: bool = False, x_step: int | None = None, out_step: int | None = None, tile: int | None = None,
                 splits: int | None = None) -> torch.Tensor:
        """``x [M, cols]``.  ``table`` (``[vocabulary, rows]``) with ``ids [M]``: the result is ``gelu_tanh(y) * table[ids]``;
        ``softcap`` c > 0: ``c tanh(y / c)``; ``add_to``: ``scale * y`` is added to this fp32 stream, which is also the result;
        ``fp32``: the result stays fp32.  Groups: matrix g reads ``x`` from column ``g * x_step`` (by default ``cols``) and writes
        ``out`` from column ``g * out_step`` (by default ``out_width``)."""
        m, n, k, g = x.shape[0], self.w.shape[0] // self.groups, self.w.shape[1], self.groups
        assert x.shape[1] == g * k if x_step is None else x.shape[1] >= (g - 1) * x_step + k
        x_step, out_step = k if x_step is None else x_step, self.out_width if out_step is None else out_step
        assert x.stride(1) == 1 and x.dtype == self.w.dtype and self.w.is_contiguous()
        width = (g - 1) * out_step + self.out_width
        if add_to is not None:
            assert self.glu is None and add_to.dtype == torch.float32 and add_to.shape == (m, width) and add_to.stride(1) == 1
            out = add_to
        elif out is None:
            out = torch.empty((m, width), dtype=torch.float32 if fp32 else x.dtype, device=x.device)
        else:
            assert out.shape[0] == m and out.shape[1] >= width and out.stride(1) == 1 and out.dtype == (torch.float32 if fp32 else x.dtype)
        kind, alpha, limit = BIAS, 0.0, 0.0
        if isinstance(self.glu, str):
            kind = UNITS[self.glu]
        elif self.glu is not None:
            kind, (alpha, limit) = GLU, self.glu
        elif self.act is not None:
            assert add_to is None and not fp32 and table is None and softcap == 0
            kind = ACTIVATIONS[self.act]
        elif add_to is not None:
            kind, alpha = ADD, scale
        elif fp32:
            kind = FLOAT
        elif softcap > 0:
            kind, limit = SOFTCAP, softcap
        elif table is not None:
            assert table.shape[1] == n and table.is_contiguous() and table.dtype == x.dtype and ids.dtype == torch.int32
            kind = GELU
        t, s = plan(m, n * g, k)
        t, s = (t if tile is None else tile), (s if splits is None else splits)
        rc = dense_lib().mfq_dense_linear(ptr(self.w), ptr(x), x.stride(0), ptr(out), out.stride(0), ptr(self.bias), m, n, k, g, x_step,
                                          out_step, kind, alpha, limit, ptr(table), ptr(ids), t, s, is_fp32(x.dtype),
                                          ptr(Workspace.get(x.device).status), stream_ptr())
        check(rc, "dense_linear")
        return out


def interleave_glu(gate: torch.Tensor, up_: torch.Tensor) -> torch.Tensor:
    """Rows of two ``[F, K]`` matrices (F a multiple of 8) as blocks of 8 gate rows followed by the 8 matching up rows."""
    f, k = gate.shape
    return torch.stack([gate.reshape(f // 8, 8, k), up_.reshape(f // 8, 8, k)], 1).reshape(2 * f, k).contiguous()


def embed_scaled(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0, copy: bool = True):
    """``(x, act)``: the fp32 stream ``table[ids] * scale`` and its copy in the activation type (the same tensor in fp32, or
    without ``copy``)."""
    t, w = ids.numel(), table.shape[1]
    x = torch.empty((t, w), dtype=torch.float32, device=table.device)
    act = None if table.dtype == torch.float32 or not copy else torch.empty((t, w), dtype=table.dtype, device=table.device)
    check(dense_lib().mfq_embed_scaled(ptr(ids), ptr(table), float(scale), ptr(x), ptr(act), t, w, is_fp32(table.dtype), stream_ptr()),
          "embed_scaled")
    return x, (x if act is None else act)


def norm_add(y: torch.Tensor, weight: torch.Tensor, x: torch.Tensor, act: torch.Tensor, width: int, eps: float) -> None:
    """In place: ``x += y / sqrt(mean(y^2) + eps) * weight`` (fp32, the mean over ``width`` columns); ``act`` follows ``x``."""
    m, w = x.shape
    assert y.shape == x.shape and y.is_contiguous() and x.dtype == torch.float32 and weight.dtype == torch.float32
    copy = None if act is x else act
    check(dense_lib().mfq_norm_add(ptr(y), ptr(weight), ptr(x), ptr(copy), m, w, width, float(eps), is_fp32(y.dtype), stream_ptr()),
          "norm_add")


def norm_out(x: torch.Tensor, weight: torch.Tensor, width: int, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps) * weight`` of the fp32 stream, in ``dtype``."""
    m, w = x.shape
    out = torch.empty((m, w), dtype=dtype, device=x.device)
    check(dense_lib().mfq_norm_out(ptr(x), ptr(weight), ptr(out), m, w, width, float(eps), is_fp32(dtype), stream_ptr()), "norm_out")
    return out


def layer_norm_out(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, width: int, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """``(x - mean) / sqrt(var + eps) * weight + bias`` of the fp32 stream (over ``width`` columns), in ``dtype``."""
    m, w = x.shape
    out = torch.empty((m, w), dtype=dtype, device=x.device)
    check(dense_lib().mfq_layer_norm_out(ptr(x), ptr(weight), ptr(bias), ptr(out), m, w, width, float(eps), is_fp32(dtype), stream_ptr()),
          "layer_norm_out")
    return out


def norm_conv_out(x: torch.Tensor, weight: torch.Tensor, conv: torch.Tensor, state: torch.Tensor | None, slots: torch.Tensor, width: int, eps: float,
                  dtype: torch.dtype, *, starts: torch.Tensor | None = None, max_q: int = 1, singles: int = 0) -> torch.Tensor:
    """``h + conv(h)`` in ``dtype``, ``h = x / sqrt(mean(x^2) + eps) * weight`` of the fp32 stream and a causal convolution over time per
    channel (``conv [taps, W]``, last row for the current token).  ``state [slots, taps - 1, W]`` fp32 keeps every sequence's last rows
    ``h`` (None with one tap); ``starts [B + 1]``: first row of every portion, whose first ``singles`` have one, or None for one row per
    sequence; ``max_q``: the longest portion."""
    out = torch.empty(x.shape, dtype=dtype, device=x.device)

    def run(seqs, first, longest):
        check(dense_lib().mfq_norm_conv(ptr(x), ptr(weight), ptr(conv), ptr(state), ptr(seqs), ptr(first), ptr(out), seqs.numel(), longest, x.shape[0],
                                        x.shape[1], width, conv.shape[0], float(eps), is_fp32(dtype), stream_ptr()), "norm_conv")
    singles = slots.numel() if starts is None else singles
    if singles:
        run(slots[:singles], None, 1)
    if singles < slots.numel():
        run(slots[singles:], starts[singles:], max_q)
    return out

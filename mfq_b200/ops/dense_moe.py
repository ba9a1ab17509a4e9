"""Mixture-of-experts feed-forward of the unquantized path (``csrc/moe_route.cu``, ``csrc/dense_moe.cu``, expert form of
``csrc/dense_gemm.cu``).

Router logits stay in fp32.  The routes of a batch are sorted by expert; few of them stream the chosen experts' weights straight
against the unsorted rows, more run tcgen05 tiles over a sorted copy.  The experts' outputs are added to the fp32 stream.
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .dense import SILU_GLU, BIAS, DenseLinear, is_fp32
from .lib import Workspace, check, dense_lib, ptr, stream_ptr

STREAM_ROUTES = 256  # batches of up to so many routes take the weight-streaming kernel


@dataclass
class ExpertBank:
    """``experts`` gated units ``down (silu(gate) * up)``: ``gate_up [experts * 2 F, W]`` (rows of each expert interleaved as by
    :func:`~mfq_b200.ops.dense.interleave_glu`), ``down [experts * W, F]``."""

    experts: int
    gate_up: torch.Tensor
    down: torch.Tensor


@dataclass
class Router:
    """``top`` experts by ``sigmoid(logit) + correction``; their weights are the sigmoids, normalised, times ``scale``."""

    linear: DenseLinear  # rows of the experts, padded to a multiple of 16
    correction: torch.Tensor  # [experts] fp32
    experts: int
    top: int
    scale: float

    def __call__(self, h: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
        return topk(self.linear(h, fp32=True)[:, : self.experts].contiguous(), self.top, self.correction, self.scale)


@dataclass
class Routes:
    offsets: torch.Tensor  # [experts + 1] first sorted row of every expert
    dest: torch.Tensor  # [T, top] sorted row of every route
    source: torch.Tensor  # [T * top] token of every sorted row
    tiles: torch.Tensor  # [entries, 2] (expert, tile), (-1, -1) where unused
    totals: torch.Tensor
    tile: int


def topk(logits: torch.Tensor, top: int, correction: torch.Tensor | None, scale: float) -> tuple[torch.Tensor, torch.Tensor]:
    t, e = logits.shape
    ids = torch.empty((t, top), dtype=torch.int32, device=logits.device)
    weight = torch.empty((t, top), dtype=torch.float32, device=logits.device)
    check(dense_lib().mfq_moe_topk(ptr(logits), ptr(correction), ptr(ids), ptr(weight), t, e, top, 1, 1, float(scale), stream_ptr()), "moe_topk")
    return ids, weight


def routes(ids: torch.Tensor, experts: int, tile: int) -> Routes:
    t, top = ids.shape
    n, dev = t * top, ids.device
    entries = min(n, math.ceil(n / tile) + min(experts, n))
    i32 = lambda *shape: torch.empty(shape, dtype=torch.int32, device=dev)
    r = Routes(i32(experts + 1), i32(t, top), i32(n), i32(entries, 2), i32(2), tile)
    check(dense_lib().mfq_moe_plan(ptr(ids), t, top, 0, experts, tile, ptr(r.offsets), ptr(r.dest), ptr(r.source), ptr(r.tiles), entries,
                                   ptr(r.totals), stream_ptr()), "moe_plan")
    return r


def token_tile(routes_: int, experts: int, fp32: bool) -> int:
    """Rows per tile for a batch of so many routes; 0: the streaming kernel."""
    if fp32:
        return 64
    if routes_ <= STREAM_ROUTES:
        return 0
    mean = routes_ / experts
    return next((b for b in (16, 32, 64) if mean <= b), 128)


def _product(w: torch.Tensor, x: torch.Tensor, r: Routes, experts: int, rows: int, kind: int, tile: int, gather: bool) -> torch.Tensor:
    n, k = w.shape[0] // experts, w.shape[1]
    out = torch.empty((rows, n // 2 if kind == SILU_GLU else n), dtype=x.dtype, device=x.device)
    rc = dense_lib().mfq_dense_experts(ptr(w), ptr(x), x.stride(0), ptr(out), out.stride(0), x.shape[0], n, k, experts, ptr(r.tiles),
                                       r.tiles.shape[0], ptr(r.offsets), ptr(r.source) if gather else None, kind,
                                       0 if tile == 0 else r.tile, is_fp32(x.dtype), ptr(Workspace.get(x.device).status), stream_ptr())
    check(rc, "dense_experts")
    return out


def add_experts(h: torch.Tensor, ids: torch.Tensor, weight: torch.Tensor, bank: ExpertBank, x: torch.Tensor, scale: float,
                tile: int | None = None) -> None:
    """``x += scale * sum_k weight[:, k] * expert_{ids[:, k]}(h)``; ``h [T, W]``, ``x [T, W]`` fp32."""
    t, top = ids.shape
    rows, fp32 = t * top, h.dtype == torch.float32
    tile = token_tile(rows, bank.experts, fp32) if tile is None else tile
    r = routes(ids, bank.experts, tile or 16)
    if tile:
        sorted_ = torch.empty((rows, h.shape[1]), dtype=h.dtype, device=h.device)
        check(dense_lib().mfq_moe_rows_sorted(ptr(h), ptr(r.source), ptr(r.totals), ptr(sorted_), rows, h.shape[1] * h.element_size(),
                                              h.stride(0) * h.element_size(), stream_ptr()), "moe_rows_sorted")
        h = sorted_
    y = _product(bank.gate_up, h, r, bank.experts, rows, SILU_GLU, tile, gather=not tile)
    y = _product(bank.down, y, r, bank.experts, rows, BIAS, tile, gather=False)
    check(dense_lib().mfq_moe_add_experts(ptr(y), ptr(r.dest), ptr(weight), ptr(x), t, x.shape[1], top, float(scale), int(fp32), stream_ptr()),
          "moe_add_experts")

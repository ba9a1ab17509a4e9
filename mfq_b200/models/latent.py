"""What models with latent attention over unquantized pages share (:mod:`~mfq_b200.ops.latent_attn`): the expansions of a layer and
the choice between attending in latent space and over expanded keys and values.

A layer's specification brings ``heads, dim, rot_dim, vdim, kv_rank, window, scale``.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops import latent_attn, window_attn
from ..ops.dense import DenseLinear, up
from .llama import StepBuffers
from .unquantized import TensorReader, fit


@dataclass
class LatentUp:
    absorb: DenseLinear  # per head [rank, dim]: queries into latent space
    value_up: DenseLinear  # per head [vdim, rank]
    expand: torch.Tensor | None  # per head [dim | rot | vdim, rank + rot]: a row of the cache to keys and values (bf16)

    @classmethod
    def read(cls, r: TensorReader, m, p: str) -> "LatentUp":
        """From the tensors ``<p>key_up.weight`` and ``<p>value_up.weight``."""
        h, d, rot, e, rank = m.heads, up(m.dim), up(m.rot_dim), up(m.vdim), up(m.kv_rank)
        uk = r.heads(p + "key_up.weight", h, m.dim, d, m.kv_rank, rank)
        uv = r.heads(p + "value_up.weight", h, m.vdim, e, m.kv_rank, rank)
        expand = None
        if r.dtype == torch.bfloat16:
            expand = torch.zeros((h, d + rot + e, rank + rot), dtype=r.dtype, device=r.device)
            expand[:, :d, :rank], expand[:, d + rot :, :rank] = uk, uv
            expand[:, d : d + rot, rank:] = torch.eye(rot, dtype=r.dtype, device=r.device)
            expand = expand.reshape(-1, rank + rot)
        return cls(DenseLinear(uk.transpose(1, 2).reshape(-1, d).contiguous(), groups=h), DenseLinear(uv.reshape(-1, rank).contiguous(), groups=h), expand)


def check_sizes(m) -> None:
    """Raises for a layer the kernels have no room for."""
    if min(m.heads, m.dim, m.vdim, m.kv_rank) < 1 or m.rot_dim < 0 or m.rot_dim % 2 or not m.scale > 0 or m.window < 1:
        raise ValueError(f"unsupported latent attention {m}")
    if up(m.kv_rank) > latent_attn.MAX_RANK or up(m.kv_rank) + up(m.rot_dim) > latent_attn.MAX_ROW:
        raise ValueError(f"latents above {latent_attn.MAX_RANK} channels are not supported")
    if up(m.dim) + up(m.rot_dim) > window_attn.MAX_HEAD or m.vdim > window_attn.MAX_HEAD:
        raise ValueError(f"heads above {window_attn.MAX_HEAD} channels are not supported")


def head_rows(q: torch.Tensor, m, width: int) -> torch.Tensor:
    """A query projection ``[heads * (dim + rot_dim), cols]`` in the stored layout ``[heads * (up(dim) + up(rot_dim)), width]``."""
    q = q.reshape(m.heads, m.dim + m.rot_dim, -1)
    return torch.cat([fit(q[:, : m.dim], m.heads, up(m.dim), width), fit(q[:, m.dim :], m.heads, up(m.rot_dim), width)], 1).reshape(-1, width)


def attend(model, m, w: LatentUp, proj: torch.Tensor, pages: torch.Tensor, step: StepBuffers, prefill: bool, *, rope, own_rows: bool,
           norm: torch.Tensor | None = None, sink: torch.Tensor | None = None) -> torch.Tensor:
    """``proj [T, heads * (dim + rot) ...]``: queries, and with ``own_rows`` the shared rows behind them, which are normed (``norm``) and
    written to ``pages`` first.  Returns the heads' outputs ``[T, heads * vdim]`` (widths as stored)."""
    t, heads, d, rot, e, rank = proj.shape[0], m.heads, up(m.dim), up(m.rot_dim), up(m.vdim), up(m.kv_rank)
    fp32 = proj.dtype == torch.float32
    singles = step.num_decode if prefill else t
    latent_rows = t if fp32 or step.max_q < latent_attn.EXPAND_MIN_TOKENS else singles
    q_latent, q = latent_attn.finish(proj, pages if own_rows else None, step.positions, step.slots, heads=heads, d=d, rank=rank, rot=rot,
                                     real_rank=m.kv_rank, real_rot=m.rot_dim, norm_w=norm, rope=rope, eps=model.cfg.norm_eps, latent_rows=latent_rows)
    y = torch.empty((t, heads * e), dtype=proj.dtype, device=proj.device)
    if latent_rows:
        w.absorb(proj[:latent_rows], x_step=d + rot, out=q_latent.view(latent_rows, -1), out_step=rank + rot)
        how = dict(rank=rank, window=m.window, scale=m.scale, sink=sink)
        if fp32:
            a = latent_attn.plain(q_latent, pages, step.block_table, model._sequence_of_rows(step, t), step.positions, **how)
        else:
            each = latent_rows > singles  # several rows of a sequence
            how["splits"] = min(model.attn_splits, latent_attn.decode_splits(latent_rows, heads, m.window))
            a = latent_attn.decode(q_latent, pages, step.block_table, step.positions if each else step.seq_lens,
                                   tok_seq=step.tok_seq if each else None, **how)
        w.value_up(a.view(latent_rows, -1), out=y[:latent_rows])
    if latent_rows < t:
        _attend_expanded(m, w, q, pages, step, singles, sink, y.view(t, heads, e))
    return y


def _attend_expanded(m, w: LatentUp, q, pages, step: StepBuffers, singles: int, sink, y) -> None:
    """Portions of the sequences from ``singles`` on, over keys and values expanded from the visible rows."""
    table, dk, dv = step.block_table[singles:], q.shape[-1], y.shape[-1]
    if m.window not in step.plans:
        seq, shift = latent_attn.visible_pages(step.portions[singles:], m.window)
        both = torch.tensor(seq + shift, dtype=torch.int32).pin_memory().to(q.device, non_blocking=True)
        step.plans[m.window] = both.split([len(seq), len(shift)])
    seq, shift = step.plans[m.window]
    rows = latent_attn.visible_rows(pages, table, seq, shift)
    group = max(1, min(m.heads, latent_attn.EXPANDED_BYTES // (rows.shape[0] * (dk + dv) * 2)))
    for h0 in range(0, m.heads, group):
        n = min(group, m.heads - h0)
        kv = DenseLinear(w.expand[h0 * (dk + dv) : (h0 + n) * (dk + dv)])(rows)
        latent_attn.prefill_rows(q, kv, shift, step.q_starts[singles:], step.seq_lens[singles:], step.max_q, head0=h0, heads=n, dk=dk, dv=dv,
                                 window=m.window, scale=m.scale, sink=sink, out=y)


def decode_splits(specs, batch: int, longest: int) -> int:
    """Most KV splits a decode step takes in any of the layers ``specs``."""
    return max((latent_attn.decode_splits(batch, m.heads, min(longest, m.window)) for m in specs), default=1)

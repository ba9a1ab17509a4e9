"""What the families of the unquantized path (bf16 or fp32, ragged batches, CUDA only) share: packing of weights into the padded
layouts of the kernels, random tensors, the page cache with its rotation tables, and the base class of their models."""

from __future__ import annotations

import torch

from ..engine.kv_cache import PlainPagedKVCache
from ..engine.recurrent_state import LayerStates
from ..ops import dense, window_attn
from ..ops.dense import DenseLinear
from .llama import LlamaModel


def fit(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` in the leading corner of a zero tensor of ``shape``."""
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class TensorReader:
    """Checkpoint tensors (canonical name -> anything ``formats.dequantize`` reads, or a torch tensor) in the kernels' form."""

    def __init__(self, tensors, device, dtype: torch.dtype) -> None:
        dense.is_fp32(dtype)
        self.tensors, self.device, self.dtype = tensors, torch.device(device), dtype

    def get(self, name: str) -> torch.Tensor:
        from .moe_decoder import _to_float
        t = self.tensors[name]
        return t.to(self.device) if isinstance(t, torch.Tensor) else _to_float(t, self.device)

    def vec(self, name: str, n: int, offset: float = 0.0) -> torch.Tensor:
        """fp32 vector plus ``offset``, zero padded to ``n``."""
        return fit(self.get(name).float().reshape(-1) + offset, n).contiguous()

    def matrix(self, name: str, rows: int, cols: int) -> torch.Tensor:
        return fit(self.get(name).to(self.dtype), rows, cols).contiguous()

    def linear(self, name: str, rows: int, cols: int, bias: bool = False) -> DenseLinear:
        return DenseLinear(self.matrix(name + ".weight", rows, cols), self.vec(name + ".bias", rows) if bias else None)

    def heads(self, name: str, heads: int, dim: int, stored: int, cols: int, width: int) -> torch.Tensor:
        """A projection to ``heads`` x ``dim`` rows as ``[heads, stored, width]``."""
        return fit(self.get(name).to(self.dtype).reshape(heads, dim, cols), heads, stored, width)

    def from_heads(self, name: str, rows: int, width: int, heads: int, dim: int, stored: int) -> torch.Tensor:
        """A projection from ``heads`` x ``dim`` channels as ``[width, heads * stored]``."""
        t = self.get(name).to(self.dtype).reshape(rows, heads, dim)
        return fit(t, width, heads, stored).reshape(width, heads * stored).contiguous()

    def glu(self, prefix: str, ff: int, cols: int, kind) -> DenseLinear:
        gate, up_ = (self.matrix(prefix + n + ".weight", ff, cols) for n in ("gate", "up"))
        return DenseLinear(dense.interleave_glu(gate, up_), glu=kind)


class RandomTensors:
    """Seeded N(0, std) tensors under canonical names, drawn when they are asked for (no second copy of a large model)."""

    def __init__(self, shapes: dict[str, tuple[int, ...]], device, seed: int = 0, std: float = 0.02, near_one=()) -> None:
        """``near_one``: name endings whose tensors are 1 + 0.1 N(0, 1)."""
        self.shapes, self.device, self.std, self.near_one = shapes, torch.device(device), std, tuple(near_one)
        self.gen = torch.Generator(device=self.device).manual_seed(seed)

    def __getitem__(self, name: str) -> torch.Tensor:
        t = torch.randn(self.shapes[name], generator=self.gen, device=self.device, dtype=torch.float32)
        return 1 + 0.1 * t if self.near_one and name.endswith(self.near_one) else (t * self.std).to(torch.bfloat16)


class UnquantizedModel(LlamaModel):
    """Stateless forward over weights of one element type; keys and values live in a :class:`PlainPagedKVCache`.

    ``cfg`` brings ``kv_shapes()``, ``kv_token_bytes(element_bytes)``, ``rotations()`` (the ``(base, dims)`` or ``(base, dims,
    scaling)`` of its layers) and ``key_spans()`` (``(KV heads, window, kept keys)`` of its attention layers)."""

    ragged = True

    def __init__(self, cfg, weights, collective=None) -> None:
        if collective is not None:
            raise NotImplementedError("this family runs on a single rank")
        if weights.embed.device.type != "cuda":
            raise RuntimeError("this family runs on a CUDA device only")
        self.cfg, self.w, self.tp, self.collective = cfg, weights, 1, None
        self.hq, self.hk = cfg.num_heads, cfg.num_kv_heads
        self.attn_splits = 1
        self._rope: dict[tuple, torch.Tensor] = {}
        self._rows: torch.Tensor | None = None

    def kv_token_bytes(self) -> int:
        return self.cfg.kv_token_bytes(self.w.embed.element_size())

    def make_cache(self, *, num_pages: int, max_seqs: int, max_pages_per_seq: int, device) -> PlainPagedKVCache:
        cache = PlainPagedKVCache(self.cfg.kv_shapes(), self.w.dtype, num_pages=num_pages, max_seqs=max_seqs,
                                  max_pages_per_seq=max_pages_per_seq, device=device)
        n = max_pages_per_seq * cache.page_size  # positions an engine with this cache can reach
        for key in self.cfg.rotations():
            if key[1] and (key not in self._rope or self._rope[key].shape[0] < n):
                self._rope[key] = window_attn.rope_table(key[0], key[1], n, self.w.embed.device, *key[2:])
        return cache

    def decode_splits(self, batch: int, longest: int) -> int:
        """Upper bound of the KV splits of a decode step at the current contexts (every layer caps it by what it sees)."""
        return max((window_attn.decode_splits(batch, heads, window_attn.visible_keys(longest, window, keep))
                    for heads, window, keep in self.cfg.key_spans()), default=1)

    def _sequence_of_rows(self, step, t: int) -> torch.Tensor:
        """Row -> sequence; a decode step has one row per sequence."""
        if step.tok_seq is not None:
            return step.tok_seq
        if self._rows is None or self._rows.numel() < t:
            self._rows = torch.arange(max(t, 256), dtype=torch.int32, device=self.w.embed.device)
        return self._rows[:t]


class RecurrentModel(UnquantizedModel):
    """Models some of whose layers carry a state per sequence: ``cfg`` also brings ``state_shapes()`` (layer, or (layer, part), -> shape)
    and ``state_bytes()``."""

    state: LayerStates | None = None

    def make_state(self, slots: int) -> LayerStates | None:
        """Recurrent state for ``slots`` sequences (None if no layer has one)."""
        shapes = self.cfg.state_shapes()
        self.state = LayerStates(shapes, slots, self.w.embed.device) if shapes else None
        return self.state

    def state_bytes_per_row(self) -> int:
        return self.cfg.state_bytes()

"""Tepetar: a decoder with sliding-window attention, output-normalised sublayers and a per-layer token table, in bf16 or fp32.

For layer ``i`` with the fp32 stream ``x`` (sublayers read ``x`` itself, their OUTPUT is normalised):

* attention: ``q, k, v`` from one product with bias; per-head RMS norm of q and k; rotation of the leading channels; scores
  ``cap tanh(q . k scale / cap)``; a query at position p sees the ``window`` positions up to p; in layers with value mixing
  (all but the first of them) the cached value is ``(1 - lambda) v + lambda v'`` with ``v'`` that first layer's value of the
  same token;  ``x += (1 + w) rms(o)``;
* feed-forward (a layer may have none): ``g sigmoid(1.702 g) (u + 1)`` with ``g = min(gate, limit)``, ``u`` clamped to
  ``+-limit``;  ``x += (1 + w) rms(y)``;
* token side: ``y = P (gelu(G x) * e_i[token])`` with the layer's own table ``e_i``;  ``x += w rms(y)``.

Layers may differ in every size and constant (:class:`LayerSpec`).  The kernels are the unquantized path of ``ops``
(:mod:`~mfq_b200.ops.dense`, :mod:`~mfq_b200.ops.window_attn`); batches are ragged (:attr:`TepetarModel.ragged`): one forward
takes portions of prompts beside single decoded tokens.  Runs on a CUDA device only.
"""

from __future__ import annotations

from dataclasses import asdict, dataclass, field

import torch

from ..ops import dense, window_attn
from ..ops.dense import DenseLinear, up
from ..utils.profiler import scope
from . import unquantized
from .llama import StepBuffers
from .unquantized import TensorReader, UnquantizedModel, fit

GLU_ALPHA = 1.702


@dataclass(frozen=True)
class LayerSpec:
    heads: int
    kv_heads: int
    dim: int  # query / key channels per head
    vdim: int  # value channels per head
    window: int
    rot_dims: int
    rot_base: float
    scale: float
    softcap: float  # 0: none
    v_mix: bool
    ff: int  # 0: no feed-forward
    limit: float


@dataclass
class TepetarConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    embed_scale: float = 1.0
    norm_eps: float = 1e-6
    side_dim: int = 0  # 0: no token side input
    name: str = "tepetar"

    def __post_init__(self):
        self.layers = [l if isinstance(l, LayerSpec) else LayerSpec(**l) for l in self.layers]
        mixed = {(l.kv_heads, l.vdim) for l in self.layers if l.v_mix}
        if len(mixed) > 1:
            raise ValueError(f"layers that share values need the same value heads, got {sorted(mixed)}")
        for i, l in enumerate(self.layers):
            if l.heads % l.kv_heads or max(l.dim, l.vdim) > window_attn.MAX_HEAD or l.rot_dims % 2 or l.rot_dims > l.dim:
                raise ValueError(f"layer {i}: unsupported attention geometry {l}")
            if not l.scale > 0 or l.window < 1:
                raise ValueError(f"layer {i}: scale and window must be positive")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_heads(self) -> int:
        return max(l.heads for l in self.layers)

    @property
    def num_kv_heads(self) -> int:
        return max(l.kv_heads for l in self.layers)

    @property
    def head_dim(self) -> int:
        return max(max(l.dim, l.vdim) for l in self.layers)

    @property
    def intermediate_size(self) -> int:
        return max(l.ff for l in self.layers)

    @classmethod
    def from_source(cls, src: dict) -> "TepetarConfig":
        """The model's own ``config.json``."""
        layers = []
        for i, entry in enumerate(src["layers"]):
            if entry.get("type") != "attention":
                raise ValueError(f"layer {i}: unknown mixer {entry.get('type')!r}")
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            rot, mask = m.get("rot") or {}, m.get("mask") or {}
            layers.append(LayerSpec(
                heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                window=min(int(mask.get("size") or window_attn.NO_WINDOW), window_attn.NO_WINDOW),
                rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)), scale=float(m["scale"]),
                softcap=float(m.get("softcap") or 0.0), v_mix=bool(m.get("v_mix", False)),
                ff=int(mlp["ff"]) if mlp is not None else 0, limit=float(mlp["limit"]) if mlp is not None else 0.0))
        return cls(vocab_size=int(src["vocab"]), hidden_size=int(src["width"]), layers=layers,
                   embed_scale=float(src["embedding"]["scale"]), norm_eps=float(src["norm"]["eps"]),
                   side_dim=int((src.get("token_side") or {}).get("dim", 0)))

    def to_dict(self) -> dict:
        """The form checkpoints carry: this class's fields plus the summary keys other tools read."""
        return {**asdict(self), "family": "tepetar", "num_layers": self.num_layers, "num_heads": self.num_heads,
                "num_kv_heads": self.num_kv_heads, "head_dim": self.head_dim, "intermediate_size": self.intermediate_size}

    @classmethod
    def from_dict(cls, raw: dict) -> "TepetarConfig":
        return cls(**{k: v for k, v in raw.items() if k in cls.__dataclass_fields__})

    @classmethod
    def uniform(cls, *, vocab_size: int, hidden_size: int, num_layers: int, heads: int, kv_heads: int, dim: int, vdim: int,
                window: int, ff: int, side_dim: int, rot_dims: int | None = None, rot_base: float = 5e5, softcap: float = 50.0,
                limit: float = 7.0, v_mix: bool = True, embed_scale: float = 1.0, norm_eps: float = 1e-6,
                name: str = "tepetar") -> "TepetarConfig":
        """All layers alike (benchmarks)."""
        layer = LayerSpec(heads, kv_heads, dim, vdim, window, dim if rot_dims is None else rot_dims, rot_base, dim ** -0.5, softcap,
                          v_mix, ff, limit)
        return cls(vocab_size, hidden_size, [layer] * num_layers, embed_scale, norm_eps, side_dim, name)

    def kv_shapes(self) -> list[tuple[int, int, int]]:
        """Per layer: (KV heads, stored key width, stored value width)."""
        return [(l.kv_heads, up(l.dim), up(l.vdim)) for l in self.layers]

    def rotations(self) -> set[tuple[float, int]]:
        return {(l.rot_base, l.rot_dims) for l in self.layers}

    def key_spans(self) -> list[tuple[int, int, int]]:
        """Per layer: (KV heads, window, kept first keys)."""
        return [(l.kv_heads, l.window, 0) for l in self.layers]

    def kv_token_bytes(self, element_bytes: int) -> int:
        return sum(g * (dk + dv) for g, dk, dv in self.kv_shapes()) * element_bytes

    def param_count(self) -> int:
        h, total = self.hidden_size, 2 * self.vocab_size * self.hidden_size
        for l in self.layers:
            total += h * (l.heads * l.dim + l.kv_heads * (l.dim + l.vdim) + l.heads * l.vdim) + 3 * h * l.ff
            total += self.side_dim * (2 * h + self.vocab_size)
        return total


@dataclass
class TepetarLayer:
    qkv: DenseLinear  # rows q | k | v, every head padded to a multiple of 16 channels
    q_norm: torch.Tensor  # [dk] fp32
    k_norm: torch.Tensor
    value_mix: float
    o_proj: DenseLinear
    attn_post_norm: torch.Tensor  # [W] fp32, the factor itself (1 + stored)
    gate_up: DenseLinear | None
    down: DenseLinear | None
    mlp_post_norm: torch.Tensor | None
    side_gate: DenseLinear | None
    side_table: torch.Tensor | None  # [V, side] this layer's slice of the token table
    side_proj: DenseLinear | None
    side_norm: torch.Tensor | None


class TepetarWeights:
    """Weights in the layout the kernels read (widths rounded up, padding zero), on one device in one element type."""

    tp_rank, tp_size, mtp = 0, 1, None

    def __init__(self, cfg: TepetarConfig, tensors, device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``tensors``: canonical name -> checkpoint tensor (anything ``formats.dequantize`` reads, or a torch tensor)."""
        r = TensorReader(tensors, device, dtype)
        self.dtype = dtype
        w = up(cfg.hidden_size)
        get, vec, linear = r.get, r.vec, r.linear
        self.embed = r.matrix("model.token_embedding.weight", cfg.vocab_size, w)
        self.lm_head = linear("model.output", up(cfg.vocab_size), w)
        self.final_norm = vec("model.output_norm.weight", w, 1.0)
        side, sp = cfg.side_dim, up(cfg.side_dim)
        table = get("model.token_side.embedding.weight") if side else None
        self.layers: list[TepetarLayer] = []
        for i, l in enumerate(cfg.layers):
            p = f"model.block.{i}."
            dk, dv = up(l.dim), up(l.vdim)
            parts, biases = [], []
            for name, heads, d, dp in (("query", l.heads, l.dim, dk), ("key", l.kv_heads, l.dim, dk), ("value", l.kv_heads, l.vdim, dv)):
                parts.append(r.heads(p + f"attention.{name}.weight", heads, d, dp, cfg.hidden_size, w).reshape(heads * dp, w))
                biases.append(fit(get(p + f"attention.{name}.bias").float().reshape(heads, d), heads, dp).reshape(-1))
            o_proj = DenseLinear(r.from_heads(p + "attention.output.weight", cfg.hidden_size, w, l.heads, l.vdim, dv),
                                 vec(p + "attention.output.bias", w))
            gate_up = down = mlp_norm = None
            if l.ff:
                fp = up(l.ff, 8)
                gate_up = r.glu(p + "mlp.", fp, w, (GLU_ALPHA, l.limit))
                down, mlp_norm = linear(p + "mlp.down", w, fp), vec(p + "mlp.post_norm.weight", w, 1.0)
            side_w = [None] * 4
            if side:
                side_w = [linear(p + "token_side.gate", sp, w),
                          fit(table[:, i * side : (i + 1) * side].to(dtype), cfg.vocab_size, sp).contiguous(),
                          linear(p + "token_side.projection", w, sp), vec(p + "token_side.norm.weight", w)]
            self.layers.append(TepetarLayer(
                DenseLinear(torch.cat(parts).contiguous(), torch.cat(biases).contiguous()), vec(p + "attention.query_norm.weight", dk),
                vec(p + "attention.key_norm.weight", dk), float(get(p + "attention.value_mix")), o_proj,
                vec(p + "attention.post_norm.weight", w, 1.0), gate_up, down, mlp_norm, *side_w))

    def nbytes(self) -> int:
        from .hybrid import _tensor_bytes
        return _tensor_bytes([self.embed, self.lm_head, self.final_norm, self.layers])


def tensor_shapes(cfg: TepetarConfig) -> dict[str, tuple[int, ...]]:
    """Canonical names and shapes of a checkpoint of this design."""
    h, out = cfg.hidden_size, {}
    out["model.token_embedding.weight"] = out["model.output.weight"] = (cfg.vocab_size, h)
    out["model.output_norm.weight"] = (h,)
    if cfg.side_dim:
        out["model.token_side.embedding.weight"] = (cfg.vocab_size, cfg.num_layers * cfg.side_dim)
    for i, l in enumerate(cfg.layers):
        p = f"model.block.{i}."
        for name, n in (("query", l.heads * l.dim), ("key", l.kv_heads * l.dim), ("value", l.kv_heads * l.vdim)):
            out[p + f"attention.{name}.weight"], out[p + f"attention.{name}.bias"] = (n, h), (n,)
        out[p + "attention.query_norm.weight"] = out[p + "attention.key_norm.weight"] = (l.dim,)
        out[p + "attention.value_mix"] = ()
        out[p + "attention.output.weight"], out[p + "attention.output.bias"] = (h, l.heads * l.vdim), (h,)
        out[p + "attention.post_norm.weight"] = (h,)
        if l.ff:
            out[p + "mlp.gate.weight"] = out[p + "mlp.up.weight"] = (l.ff, h)
            out[p + "mlp.down.weight"], out[p + "mlp.post_norm.weight"] = (h, l.ff), (h,)
        if cfg.side_dim:
            out[p + "token_side.gate.weight"], out[p + "token_side.projection.weight"] = (cfg.side_dim, h), (h, cfg.side_dim)
            out[p + "token_side.norm.weight"] = (h,)
    return out


class RandomTensors(unquantized.RandomTensors):
    """Seeded random tensors of a configuration."""

    def __init__(self, cfg: TepetarConfig, device, seed: int = 0, std: float = 0.02) -> None:
        super().__init__(tensor_shapes(cfg), device, seed, std, ("query_norm.weight", "key_norm.weight", "token_side.norm.weight"))


class TepetarModel(UnquantizedModel):
    def __init__(self, cfg: TepetarConfig, weights: TepetarWeights, collective=None) -> None:
        super().__init__(cfg, weights, collective)
        mixed = [i for i, l in enumerate(cfg.layers) if l.v_mix]
        self.first_mixed = mixed[0] if mixed else -1

    # -- forward ----------------------------------------------------------------------------------------------------
    def _attend(self, q, kv, l: LayerSpec, step: StepBuffers, prefill: bool):
        t = q.shape[0]
        how = dict(window=l.window, scale=l.scale, cap=l.softcap)
        if q.dtype == torch.float32:
            return window_attn.plain(q, kv, step.block_table, self._sequence_of_rows(step, t), step.positions, **how)
        singles = step.num_decode if prefill else t
        out = torch.empty((t, l.heads, kv.v.shape[-1]), dtype=q.dtype, device=q.device)
        if singles:
            splits = min(self.attn_splits, window_attn.decode_splits(singles, l.kv_heads, l.window))
            window_attn.decode(q[:singles], kv, step.block_table[:singles], step.seq_lens[:singles], splits=splits,
                               out=out[:singles], **how)
        if prefill and singles < step.seq_lens.numel():
            window_attn.prefill(q, kv, step.block_table[singles:], step.q_starts[singles:], step.seq_lens[singles:], step.max_q,
                                out=out, **how)
        return out

    def _block_at(self, i: int, x, act, cache, step: StepBuffers, prefill: bool, v_first):
        """Layer ``i`` over the stream ``x`` (in place; ``act`` is its copy in the activation type)."""
        cfg, l, w = self.cfg, self.cfg.layers[i], self.w.layers[i]
        kv = cache.layer(i)
        dk, dv = kv.k.shape[-1], kv.v.shape[-1]
        with scope("attn.qkv", x.device):
            qkv = w.qkv(act)
        with scope("attn.core", x.device):
            mixes = l.v_mix and i != self.first_mixed
            q = window_attn.qkv_finish(
                qkv, kv, step.positions, step.slots, heads=l.heads, kv_heads=l.kv_heads, dim=l.dim, q_norm=w.q_norm, k_norm=w.k_norm,
                rope=self._rope.get((l.rot_base, l.rot_dims)), rot=l.rot_dims, eps=cfg.norm_eps, v_first=v_first if mixes else None,
                mix=w.value_mix if mixes else 0.0)
            if i == self.first_mixed:
                v_first = qkv[:, (l.heads + l.kv_heads) * dk :]
            o = self._attend(q, kv, l, step, prefill)
        with scope("attn.o_proj", x.device):
            dense.norm_add(w.o_proj(o.view(o.shape[0], l.heads * dv)), w.attn_post_norm, x, act, cfg.hidden_size, cfg.norm_eps)
        if w.gate_up is not None:
            with scope("ffn.gate_up", x.device):
                y = w.gate_up(act)
            with scope("ffn.down", x.device):
                dense.norm_add(w.down(y), w.mlp_post_norm, x, act, cfg.hidden_size, cfg.norm_eps)
        if w.side_gate is not None:
            with scope("token_side", x.device):
                y = w.side_proj(w.side_gate(act, table=w.side_table, ids=step.input_ids))
                dense.norm_add(y, w.side_norm, x, act, cfg.hidden_size, cfg.norm_eps)
        return v_first

    def forward(self, step: StepBuffers, cache, *, prefill: bool, logits_rows: torch.Tensor | None = None,
                gather_logits: bool = True, return_hidden: bool = False, layer_outputs: list | None = None):
        """Logits ``[rows, vocab]`` in the model's element type (all tokens, or ``logits_rows`` of them).  ``prefill``: a
        ragged batch whose first ``step.num_decode`` rows are single tokens; otherwise one token per sequence.
        ``layer_outputs`` receives a copy of the fp32 stream after every layer."""
        cfg = self.cfg
        x, act = dense.embed_scaled(step.input_ids, self.w.embed, cfg.embed_scale)
        v_first = None
        for i in range(cfg.num_layers):
            v_first = self._block_at(i, x, act, cache, step, prefill, v_first)
            if layer_outputs is not None:
                layer_outputs.append(x[:, : cfg.hidden_size].clone())
        rows = x if logits_rows is None else x.index_select(0, logits_rows.long())
        with scope("head", x.device):
            h = dense.norm_out(rows, self.w.final_norm, cfg.hidden_size, cfg.norm_eps, self.w.dtype)
            logits = self.w.lm_head(h)[:, : cfg.vocab_size]
        return (logits, x) if return_hidden else logits

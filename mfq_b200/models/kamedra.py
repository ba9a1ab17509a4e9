"""Kamedra: a decoder of differential-attention and gated-linear-attention layers in any order, in bf16 or fp32.

Every sublayer reads the normalised fp32 stream, ``x += f(rms(x) w)``; a layer may have no feed-forward.

* attention: two query / key maps per head over shared values (:mod:`~mfq_b200.ops.window_attn`); the leading channels of a map
  are rotated in neighbouring pairs, with optionally scaled frequencies; a query at position p sees the ``window`` positions up
  to p and the first ``keep`` tokens; ``o = rms(a1 - lambda a2) (1 - diff)`` with one ``lambda`` per layer, from four learned
  vectors and ``diff``.  A layer with ``kv_from`` has queries only and reads the pages of that earlier layer;
* gated linear attention (:mod:`~mfq_b200.ops.gla`): a fp32 matrix state per head that decays per key channel, kept per
  sequence in the engine's recurrent state;
* feed-forward: ``W_down (gelu(gate) * up)``; logits come from the embedding table, with a soft cap.

Layers may differ in kind and in every size and constant.  Runs on a CUDA device only; batches are ragged.
"""

from __future__ import annotations

import math
from dataclasses import asdict, dataclass, field

import torch

from ..ops import dense, gla, window_attn
from ..ops.dense import DenseLinear, up
from ..ops.window_attn import NO_WINDOW, Difference, FrequencyScaling
from ..utils.profiler import scope
from . import unquantized
from .llama import StepBuffers
from .unquantized import RecurrentModel, TensorReader


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int  # channels of one query / key map
    vdim: int
    scale: float
    diff: float
    window: int = NO_WINDOW
    keep: int = 0  # first tokens that stay visible
    rot_dims: int = 0
    rot_base: float = 1.0
    rot_scaling: FrequencyScaling | None = None
    kv_from: int | None = None  # the layer whose keys and values this one reads

    @property
    def rotation(self) -> tuple:
        return self.rot_base, self.rot_dims, self.rot_scaling


@dataclass(frozen=True)
class GlaSpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 0  # of the decay projection; 0: what the checkpoint's tensors have


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | GlaSpec
    ff: int = 0  # 0: no feed-forward

    @property
    def linear(self) -> bool:
        return isinstance(self.mixer, GlaSpec)

    @classmethod
    def from_dict(cls, raw: dict) -> "LayerSpec":
        m = dict(raw["mixer"])
        if "tau" in m:
            return cls(GlaSpec(**m), raw["ff"])
        if m.get("rot_scaling"):
            m["rot_scaling"] = FrequencyScaling(**m["rot_scaling"])
        return cls(AttentionSpec(**m), raw["ff"])


@dataclass
class KamedraConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    logit_softcap: float = 0.0  # 0: none
    norm_eps: float = 1e-6
    name: str = "kamedra"

    def __post_init__(self):
        self.layers = [l if isinstance(l, LayerSpec) else LayerSpec.from_dict(l) for l in self.layers]
        for i, l in enumerate(self.layers):
            m = l.mixer
            if min(m.heads, m.dim, m.vdim) < 1 or l.ff < 0:
                raise ValueError(f"layer {i}: sizes must be positive: {m}")
            if l.linear:
                if not m.tau > 0 or m.vdim > 1024:
                    raise ValueError(f"layer {i}: unsupported linear attention {m}")
                continue
            if m.kv_heads < 1 or m.heads % m.kv_heads or m.heads // m.kv_heads > 128 or max(m.dim, m.vdim) > window_attn.MAX_HEAD:
                raise ValueError(f"layer {i}: unsupported attention geometry {m}")
            if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim:
                raise ValueError(f"layer {i}: {m.rot_dims} of {m.dim} channels cannot be rotated in pairs")
            if not m.scale > 0 or m.window < 1 or m.keep < 0:
                raise ValueError(f"layer {i}: scale and window must be positive")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, AttentionSpec) or src.kv_from is not None:
                    raise ValueError(f"layer {i}: layer {m.kv_from} has no keys and values to read")
                if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i}: its heads differ from those of layer {m.kv_from}")

    # -- what other parts of the framework ask a configuration for ------------------------------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def attention(self) -> list[AttentionSpec]:
        return [l.mixer for l in self.layers if not l.linear]

    @property
    def num_heads(self) -> int:
        return max(l.mixer.heads for l in self.layers)

    @property
    def num_kv_heads(self) -> int:
        return max((m.kv_heads for m in self.attention), default=1)

    @property
    def head_dim(self) -> int:
        return max(max(l.mixer.dim, l.mixer.vdim) for l in self.layers)

    @property
    def intermediate_size(self) -> int:
        return max(l.ff for l in self.layers)

    def owners(self) -> list[int]:
        """Layers with pages of their own, in order: place in the cache -> layer."""
        return [i for i, l in enumerate(self.layers) if not l.linear and l.mixer.kv_from is None]

    def kv_shapes(self) -> list[tuple[int, int, int]]:
        """Per layer with pages: (KV heads, stored key width of both maps, stored value width)."""
        return [(m.kv_heads, 2 * up(m.dim), up(m.vdim)) for m in (self.layers[i].mixer for i in self.owners())]

    def kv_token_bytes(self, element_bytes: int) -> int:
        return sum(g * (dk + dv) for g, dk, dv in self.kv_shapes()) * element_bytes

    def state_shapes(self) -> dict[int, tuple[int, int, int]]:
        """Recurrent layer -> (heads, stored key width, stored value width) of a sequence's fp32 state."""
        return {i: (l.mixer.heads, up(l.mixer.dim), up(l.mixer.vdim)) for i, l in enumerate(self.layers) if l.linear}

    def state_bytes(self) -> int:
        return sum(4 * math.prod(s) for s in self.state_shapes().values())

    def rotations(self) -> set[tuple]:
        return {m.rotation for m in self.attention}

    def key_spans(self) -> list[tuple[int, int, int]]:
        """Per attention layer: (KV heads, window, kept first keys)."""
        return [(m.kv_heads, m.window, m.keep) for m in self.attention]

    def param_count(self) -> int:
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    # -- forms ----------------------------------------------------------------------------------------------------------
    @classmethod
    def from_source(cls, src: dict) -> "KamedraConfig":
        """The model's own ``config.json``."""
        layers = []
        for i, entry in enumerate(src["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            if entry.get("type") == "gla":
                mixer = GlaSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))
            elif entry.get("type") == "attention":
                rot, mask = m.get("rot") or {}, m.get("mask") or {}
                sc = rot.get("scaling")
                mixer = AttentionSpec(
                    int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), float(m["diff"]),
                    window=min(int(mask.get("size") or NO_WINDOW), NO_WINDOW), keep=int(mask.get("keep_first") or 0),
                    rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)),
                    rot_scaling=FrequencyScaling(*(float(sc[k]) for k in ("factor", "low", "high", "original"))) if sc else None,
                    kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {entry.get('type')!r}")
            layers.append(LayerSpec(mixer, int(mlp["ff"]) if mlp is not None else 0))
        return cls(vocab_size=int(src["vocab"]), hidden_size=int(src["width"]), layers=layers,
                   logit_softcap=float(src.get("logit_softcap") or 0.0), norm_eps=float(src["norm"]["eps"]))

    def to_dict(self) -> dict:
        """The form checkpoints carry: this class's fields plus the summary keys other tools read."""
        return {**asdict(self), "family": "kamedra", "num_layers": self.num_layers, "num_heads": self.num_heads,
                "num_kv_heads": self.num_kv_heads, "head_dim": self.head_dim, "intermediate_size": self.intermediate_size}

    @classmethod
    def from_dict(cls, raw: dict) -> "KamedraConfig":
        return cls(**{k: v for k, v in raw.items() if k in cls.__dataclass_fields__})

    @classmethod
    def periodic(cls, *, vocab_size: int, hidden_size: int, num_layers: int, attention: AttentionSpec, linear: GlaSpec, ff: int,
                 every: int = 4, shared: bool = False, logit_softcap: float = 30.0, norm_eps: float = 1e-6,
                 name: str = "kamedra") -> "KamedraConfig":
        """Every ``every``-th layer is attention, the others linear (benchmarks); ``shared``: all attention layers but the first
        read its keys and values."""
        layers, first = [], None
        for i in range(num_layers):
            if i % every:
                layers.append(LayerSpec(linear, ff))
                continue
            layers.append(LayerSpec(AttentionSpec(**{**vars(attention), "kv_from": first if shared else None}), ff))
            first = i if first is None else first
        return cls(vocab_size, hidden_size, layers, logit_softcap, norm_eps, name)


def tensor_shapes(cfg: KamedraConfig) -> dict[str, tuple[int, ...]]:
    """Canonical names and shapes of a checkpoint of this design (decay ranks as far as the configuration knows them)."""
    h, out = cfg.hidden_size, {}
    out["model.token_embedding.weight"], out["model.output_norm.weight"] = (cfg.vocab_size, h), (h,)
    for i, l in enumerate(cfg.layers):
        m, p = l.mixer, f"model.block.{i}."
        out[p + "attention.norm.weight"] = (h,)
        if l.linear:
            p += "linear_attention."
            k, v = m.heads * m.dim, m.heads * m.vdim
            out |= {p + "query.weight": (k, h), p + "key.weight": (k, h), p + "value.weight": (v, h), p + "gate.weight": (v, h),
                    p + "output.weight": (h, v), p + "norm.weight": (m.vdim,), p + "decay_a.weight": (m.rank, h),
                    p + "decay_b.weight": (k, m.rank), p + "decay_b.bias": (k,)}
        else:
            p += "attention."
            out |= {p + "query.weight": (2 * m.heads * m.dim, h), p + "output.weight": (h, m.heads * m.vdim)}
            out |= {p + f"lambda_{n}": (m.dim,) for n in ("q1", "k1", "q2", "k2")}
            if m.kv_from is None:
                out |= {p + "key.weight": (2 * m.kv_heads * m.dim, h), p + "value.weight": (m.kv_heads * m.vdim, h)}
        if l.ff:
            p = f"model.block.{i}.mlp."
            out |= {p + "norm.weight": (h,), p + "gate.weight": (l.ff, h), p + "up.weight": (l.ff, h), p + "down.weight": (h, l.ff)}
    return out


class RandomTensors(unquantized.RandomTensors):
    """Seeded random tensors of a configuration (whose linear layers give their decay rank)."""

    def __init__(self, cfg: KamedraConfig, device, seed: int = 0, std: float = 0.02) -> None:
        super().__init__(tensor_shapes(cfg), device, seed, std, ("norm.weight",))


@dataclass
class AttentionWeights:
    qkv: DenseLinear  # rows q | k | v (q alone in a layer that reads another's pages), maps padded to multiples of 16 channels
    o_proj: DenseLinear
    difference: Difference


@dataclass
class GlaWeights:
    proj: DenseLinear  # rows q | k | v | gate | decay_a
    decay_b: torch.Tensor  # [heads * dk, rank]
    decay_bias: torch.Tensor  # [heads * dk] fp32
    norm: torch.Tensor  # [dv] fp32
    o_proj: DenseLinear
    geometry: gla.Geometry


@dataclass
class KamedraLayer:
    norm: torch.Tensor  # [W] fp32
    mixer: AttentionWeights | GlaWeights
    mlp_norm: torch.Tensor | None
    gate_up: DenseLinear | None
    down: DenseLinear | None


class KamedraWeights:
    """Weights in the layout the kernels read (widths rounded up, padding zero), on one device in one element type."""

    tp_rank, tp_size, mtp = 0, 1, None

    def __init__(self, cfg: KamedraConfig, tensors, device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``tensors``: canonical name -> checkpoint tensor (anything ``formats.dequantize`` reads, or a torch tensor)."""
        r = TensorReader(tensors, device, dtype)
        self.dtype = dtype
        w = up(cfg.hidden_size)
        self.embed = r.matrix("model.token_embedding.weight", up(cfg.vocab_size), w)
        self.lm_head = DenseLinear(self.embed)
        self.final_norm = r.vec("model.output_norm.weight", w)
        self.layers: list[KamedraLayer] = []
        for i, l in enumerate(cfg.layers):
            p = f"model.block.{i}."
            mixer = self._gla(r, cfg, l.mixer, p, w) if l.linear else self._attention(r, cfg, l.mixer, p, w)
            norm, mlp = r.vec(p + "attention.norm.weight", w), (None, None, None)
            if l.ff:
                fp = up(l.ff, 8)
                mlp = r.vec(p + "mlp.norm.weight", w), r.glu(p + "mlp.", fp, w, "gelu"), r.linear(p + "mlp.down", w, fp)
            self.layers.append(KamedraLayer(norm, mixer, *mlp))

    @staticmethod
    def _attention(r: TensorReader, cfg: KamedraConfig, m: AttentionSpec, p: str, w: int) -> AttentionWeights:
        p += "attention."
        dk, dv, g = up(m.dim), up(m.vdim), m.kv_heads
        q = r.heads(p + "query.weight", 2 * m.heads, m.dim, dk, cfg.hidden_size, w)
        # heads come as [head][map]; the kernels take [KV head][map][head of the KV head]
        parts = [q.reshape(g, m.heads // g, 2, dk, w).transpose(1, 2).reshape(-1, w)]
        if m.kv_from is None:
            parts.append(r.heads(p + "key.weight", 2 * g, m.dim, dk, cfg.hidden_size, w).reshape(-1, w))
            parts.append(r.heads(p + "value.weight", g, m.vdim, dv, cfg.hidden_size, w).reshape(-1, w))
        q1, k1, q2, k2 = (r.get(p + f"lambda_{n}").float() for n in ("q1", "k1", "q2", "k2"))
        weight = float((q1 * k1).sum().exp() - (q2 * k2).sum().exp() + m.diff)
        return AttentionWeights(DenseLinear(torch.cat(parts).contiguous()),
                                DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, dv)),
                                Difference(weight, 1.0 - m.diff, cfg.norm_eps, m.vdim))

    @staticmethod
    def _gla(r: TensorReader, cfg: KamedraConfig, m: GlaSpec, p: str, w: int) -> GlaWeights:
        p += "linear_attention."
        dk, dv = up(m.dim), up(m.vdim)
        parts = [r.heads(p + n + ".weight", m.heads, d, dp, cfg.hidden_size, w).reshape(-1, w)
                 for n, d, dp in (("query", m.dim, dk), ("key", m.dim, dk), ("value", m.vdim, dv), ("gate", m.vdim, dv))]
        rank = r.get(p + "decay_a.weight").shape[0]
        if m.rank and m.rank != rank:
            raise ValueError(f"{p}decay_a has rank {rank}, the configuration says {m.rank}")
        geo = gla.Geometry(m.heads, dk, dv, m.dim, m.vdim, up(rank), m.tau, cfg.norm_eps)
        parts.append(r.matrix(p + "decay_a.weight", geo.rank, w))
        return GlaWeights(DenseLinear(torch.cat(parts).contiguous()),
                          r.heads(p + "decay_b.weight", m.heads, m.dim, dk, rank, geo.rank).reshape(-1, geo.rank).contiguous(),
                          unquantized.fit(r.get(p + "decay_b.bias").float().reshape(m.heads, m.dim), m.heads, dk).reshape(-1).contiguous(),
                          r.vec(p + "norm.weight", dv),
                          DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, dv)), geo)

    def nbytes(self) -> int:
        from .hybrid import _tensor_bytes
        return _tensor_bytes([self.embed, self.final_norm, self.layers])


class KamedraModel(RecurrentModel):
    def __init__(self, cfg: KamedraConfig, weights: KamedraWeights, collective=None) -> None:
        super().__init__(cfg, weights, collective)
        place = {layer: n for n, layer in enumerate(cfg.owners())}
        self.pages_of = [None if l.linear else place[i if l.mixer.kv_from is None else l.mixer.kv_from] for i, l in enumerate(cfg.layers)]

    # -- forward ----------------------------------------------------------------------------------------------------
    def _attend(self, q, kv, m: AttentionSpec, d: Difference, step: StepBuffers, prefill: bool):
        t = q.shape[0]
        how = dict(window=m.window, keep=m.keep, scale=m.scale, cap=0.0)
        if q.dtype == torch.float32:
            maps = window_attn.plain(q, kv, step.block_table, self._sequence_of_rows(step, t), step.positions, maps=2, **how)
            return window_attn.difference(maps, m.kv_heads, d)
        singles = step.num_decode if prefill else t
        out = torch.empty((t, m.heads, kv.v.shape[-1]), dtype=q.dtype, device=q.device)
        if singles:
            seen = window_attn.visible_keys(NO_WINDOW, m.window, m.keep)
            splits = min(self.attn_splits, window_attn.decode_splits(singles, m.kv_heads, seen))
            window_attn.decode(q[:singles], kv, step.block_table[:singles], step.seq_lens[:singles], diff=d, splits=splits,
                               out=out[:singles], **how)
        if prefill and singles < step.seq_lens.numel():
            maps = window_attn.prefill(q, kv, step.block_table[singles:], step.q_starts[singles:], step.seq_lens[singles:], step.max_q,
                                       maps=2, **how)
            window_attn.difference(maps[singles:], m.kv_heads, d, out=out[singles:])
        return out

    def _attention_at(self, i: int, h, cache, step: StepBuffers, prefill: bool):
        m, w = self.cfg.layers[i].mixer, self.w.layers[i].mixer
        kv = cache.layer(self.pages_of[i])
        with scope("attn.qkv", h.device):
            qkv = w.qkv(h)
        with scope("attn.core", h.device):
            q = window_attn.qkv_finish(
                qkv, kv if m.kv_from is None else None, step.positions, step.slots, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim,
                dk=up(m.dim), q_norm=None, k_norm=None, rope=self._rope.get(m.rotation), rot=m.rot_dims, pairs=True, maps=2,
                eps=self.cfg.norm_eps)
            return self._attend(q, kv, m, w.difference, step, prefill).view(h.shape[0], -1)

    def _gla_at(self, i: int, h, step: StepBuffers, prefill: bool):
        w, state = self.w.layers[i].mixer, self.state.layer(i)
        with scope("gla.proj", h.device):
            proj = w.proj(h)
        args = (proj, w.decay_b, w.decay_bias, w.norm, state, step.state_slots, w.geometry)
        with scope("gla.core", h.device):
            if prefill:
                return gla.ragged(*args, step.q_starts, step.max_q, step.num_decode)
            return gla.recurrent(*args)

    def forward(self, step: StepBuffers, cache, *, prefill: bool, logits_rows: torch.Tensor | None = None,
                gather_logits: bool = True, return_hidden: bool = False, layer_outputs: list | None = None):
        """Logits ``[rows, vocab]`` in the model's element type (all tokens, or ``logits_rows`` of them).  ``prefill``: a
        ragged batch whose first ``step.num_decode`` rows are single tokens; otherwise one token per sequence.
        ``layer_outputs`` receives a copy of the fp32 stream after every layer."""
        cfg = self.cfg
        x, _ = dense.embed_scaled(step.input_ids, self.w.embed, copy=False)
        for i, (l, w) in enumerate(zip(cfg.layers, self.w.layers)):
            h = dense.norm_out(x, w.norm, cfg.hidden_size, cfg.norm_eps, self.w.dtype)
            y = self._gla_at(i, h, step, prefill) if l.linear else self._attention_at(i, h, cache, step, prefill)
            with scope("gla.o_proj" if l.linear else "attn.o_proj", x.device):
                w.mixer.o_proj(y, add_to=x)
            if w.gate_up is not None:
                with scope("ffn.gate_up", x.device):
                    y = w.gate_up(dense.norm_out(x, w.mlp_norm, cfg.hidden_size, cfg.norm_eps, self.w.dtype))
                with scope("ffn.down", x.device):
                    w.down(y, add_to=x)
            if layer_outputs is not None:
                layer_outputs.append(x[:, : cfg.hidden_size].clone())
        rows = x if logits_rows is None else x.index_select(0, logits_rows.long())
        with scope("head", x.device):
            h = dense.norm_out(rows, self.w.final_norm, cfg.hidden_size, cfg.norm_eps, self.w.dtype)
            logits = self.w.lm_head(h, softcap=cfg.logit_softcap)[:, : cfg.vocab_size]
        return (logits, x) if return_hidden else logits

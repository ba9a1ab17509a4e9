"""Gogivik: a decoder whose layers, in any order, mix by latent attention in a window, by attention in chunks with rotated values, or by
a state-space recurrence, in bf16 or fp32.

Every sublayer reads ``g = h + conv(h)``, ``h = rms(x) (1 + w)`` of the fp32 stream with a short causal convolution over time per channel
(one kernel), and adds to the stream, ``x += f(g)``; a layer may have no feed-forward.

* latent attention (:mod:`~mfq_b200.models.latent`): queries come from a normed latent of their own, keys and values from one normed
  latent per token plus one rotated key part shared by all heads; a sliding window and a sink per head;
* attention (:mod:`~mfq_b200.ops.window_attn`): a query sees the tokens of its own chunk of the sequence up to itself; queries and keys are
  normed and rotated with scaled frequencies; values are normed and rotated by their position, outputs turn back by the query's;
* state-space recurrence (:mod:`~mfq_b200.ops.ssd`): one decay per head, behind a short convolution, with a gated norm over parts of all
  heads' channels;
* feed-forward: ``W_down max(W_up g, 0)^2``; logits are scaled.

Layers may differ in kind and in every size and constant.  Runs on a CUDA device only; batches are ragged.
"""

from __future__ import annotations

import math
from dataclasses import asdict, dataclass, field

import torch

from ..ops import dense, latent_attn, ssd, window_attn
from ..ops.dense import DenseLinear, up
from ..ops.window_attn import NO_WINDOW, LinearScaling, ValueTurn
from ..utils.profiler import scope
from . import latent, unquantized
from .latent import LatentUp
from .llama import StepBuffers
from .unquantized import RecurrentModel, TensorReader, fit


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int  # unrotated query / key channels per head
    rot_dim: int  # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float = 1e4
    window: int = NO_WINDOW

    @property
    def rotation(self) -> tuple:
        return self.rot_base, self.rot_dim

    @property
    def row(self) -> int:
        """Stored width of a token's row of the cache."""
        return up(self.kv_rank) + up(self.rot_dim)


@dataclass(frozen=True)
class ChunkSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = NO_WINDOW
    rot_dims: int = 0
    rot_base: float = 1e4
    rot_factor: float = 1.0  # what the frequencies of queries and keys are divided by

    @property
    def rotation(self) -> tuple:
        return self.rot_base, self.rot_dims, LinearScaling(self.rot_factor)

    @property
    def value_rotation(self) -> tuple:
        return self.rot_base, self.vdim


@dataclass(frozen=True)
class StateSpec:
    heads: int
    groups: int
    state: int
    vdim: int
    taps: int
    norm_groups: int


MIXERS = {"latent_attention": LatentSpec, "attention": ChunkSpec, "mamba2": StateSpec}


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec | ChunkSpec | StateSpec
    ff: int = 0  # 0: no feed-forward

    @property
    def kind(self) -> str:
        return next(k for k, c in MIXERS.items() if isinstance(self.mixer, c))

    @classmethod
    def from_dict(cls, raw: dict) -> "LayerSpec":
        m = raw["mixer"]
        kind = LatentSpec if "kv_rank" in m else StateSpec if "state" in m else ChunkSpec
        return cls(kind(**m), raw["ff"])


@dataclass
class GogivikConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    conv_taps: int = 1  # of the convolution in front of every sublayer
    logit_scale: float = 1.0
    norm_eps: float = 1e-5
    name: str = "gogivik"

    def __post_init__(self):
        self.layers = [l if isinstance(l, LayerSpec) else LayerSpec.from_dict(l) for l in self.layers]
        if not 1 <= self.conv_taps <= 8:
            raise ValueError(f"convolutions of {self.conv_taps} taps are not supported")
        for i, l in enumerate(self.layers):
            try:
                self._check(l)
            except ValueError as exc:
                raise ValueError(f"layer {i}: {exc}") from None

    @staticmethod
    def _check(l: LayerSpec) -> None:
        m = l.mixer
        if l.ff < 0:
            raise ValueError(f"unsupported feed-forward {l.ff}")
        if l.kind == "latent_attention":
            latent.check_sizes(m)
            if m.q_rank < 1:
                raise ValueError(f"unsupported latent attention {m}")
        elif l.kind == "attention":
            if min(m.heads, m.kv_heads, m.dim, m.vdim) < 1 or m.heads % m.kv_heads or m.heads // m.kv_heads > 128 or not m.scale > 0 or m.chunk < 1:
                raise ValueError(f"unsupported attention {m}")
            if max(m.dim, m.vdim) > window_attn.MAX_HEAD:
                raise ValueError(f"heads above {window_attn.MAX_HEAD} channels are not supported")
            if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim or m.vdim % 2 or not m.rot_factor > 0:
                raise ValueError(f"{m.rot_dims} of {m.dim} query channels and {m.vdim} value channels cannot be rotated in pairs")
        else:
            if min(m.heads, m.groups, m.state, m.vdim, m.norm_groups) < 1 or m.heads % m.groups or m.heads * m.vdim % m.norm_groups:
                raise ValueError(f"unsupported recurrence {m}")
            if not 1 <= m.taps <= 8 or not ssd.column_split(1, m.heads, up(m.state), up(m.vdim)):
                raise ValueError(f"unsupported recurrence {m}")

    # -- what other parts of the framework ask a configuration for ------------------------------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def _of(self, kind: str) -> list:
        return [l.mixer for l in self.layers if l.kind == kind]

    @property
    def attention(self) -> list[ChunkSpec]:
        return self._of("attention")

    @property
    def latent(self) -> list[LatentSpec]:
        return self._of("latent_attention")

    @property
    def num_heads(self) -> int:
        return max(l.mixer.heads for l in self.layers)

    @property
    def num_kv_heads(self) -> int:
        return max((m.kv_heads for m in self.attention), default=1)

    @property
    def head_dim(self) -> int:
        return max(max(getattr(l.mixer, "dim", 0), l.mixer.vdim) for l in self.layers)

    @property
    def intermediate_size(self) -> int:
        return max(l.ff for l in self.layers)

    def owners(self) -> list[int]:
        """Layers with pages, in order: place in the cache -> layer."""
        return [i for i, l in enumerate(self.layers) if l.kind != "mamba2"]

    def kv_shapes(self) -> list[tuple[int, int, int]]:
        """Per layer with pages: (KV heads, stored key width, stored value width).  A latent row is the key; its values are part of it."""
        mixers = (self.layers[i].mixer for i in self.owners())
        return [(1, m.row, 0) if isinstance(m, LatentSpec) else (m.kv_heads, up(m.dim), up(m.vdim)) for m in mixers]

    def kv_token_bytes(self, element_bytes: int) -> int:
        return sum(g * (dk + dv) for g, dk, dv in self.kv_shapes()) * element_bytes

    def state_shapes(self) -> dict[tuple[int, str], tuple[int, ...]]:
        """(layer, part) -> shape of a sequence's fp32 state."""
        out = {}
        for i, l in enumerate(self.layers):
            m = l.mixer
            out[i, "input"] = (self.conv_taps - 1, up(self.hidden_size))
            if l.ff:
                out[i, "mlp_input"] = (self.conv_taps - 1, up(self.hidden_size))
            if l.kind == "mamba2":
                n, p = up(m.state), up(m.vdim)
                out[i, "state"] = (m.heads, n, p)
                out[i, "conv"] = (m.taps - 1, m.heads * p + 2 * m.groups * n)
        return out

    def state_bytes(self) -> int:
        return sum(4 * math.prod(s) for s in self.state_shapes().values())

    def rotations(self) -> set[tuple]:
        return {m.rotation for m in self.latent} | {r for m in self.attention for r in (m.rotation, m.value_rotation)}

    def key_spans(self) -> list[tuple[int, int, int]]:
        """Per attention layer over keys of its own: (KV heads, most visible keys, kept first keys)."""
        return [(m.kv_heads, m.chunk, 0) for m in self.attention]

    @property
    def attention_layers(self) -> int:
        return len(self.owners())

    def param_count(self) -> int:
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    # -- forms ----------------------------------------------------------------------------------------------------------
    @classmethod
    def from_source(cls, src: dict) -> "GogivikConfig":
        """The model's own ``config.json``."""
        ints = lambda m, *names: {n: int(m[n]) for n in names}
        size = lambda m: min(int((m.get("mask") or {}).get("size") or NO_WINDOW), NO_WINDOW)
        layers = []
        for i, entry in enumerate(src["layers"]):
            m, mlp, kind = entry["mixer"], entry.get("mlp"), entry.get("type")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            rot = m.get("rot") or {}
            if kind == "latent_attention":
                if int(rot.get("dims", 0)) != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: {rot.get('dims')} rotated channels of a rotated part of {m['rot_dim']}")
                mixer = LatentSpec(**ints(m, "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), scale=float(m["scale"]),
                                   rot_base=float(rot.get("base", 1e4)), window=size(m))
            elif kind == "attention":
                mixer = ChunkSpec(**ints(m, "heads", "kv_heads", "dim", "vdim"), scale=float(m["scale"]), chunk=size(m), rot_dims=int(rot["dims"]),
                                  rot_base=float(rot["base"]), rot_factor=float((rot.get("scaling") or {}).get("factor", 1.0)))
            elif kind == "mamba2":
                mixer = StateSpec(**ints(m, "heads", "groups", "state", "vdim", "norm_groups"), taps=int(m["conv"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            layers.append(LayerSpec(mixer, int(mlp["ff"]) if mlp is not None else 0))
        return cls(vocab_size=int(src["vocab"]), hidden_size=int(src["width"]), layers=layers, conv_taps=int(src["canon"]["taps"]),
                   logit_scale=float(src["logit_scale"]), norm_eps=float(src["norm"]["eps"]))

    def to_dict(self) -> dict:
        """The form checkpoints carry: this class's fields plus the summary keys other tools read."""
        return {**asdict(self), "family": "gogivik", "num_layers": self.num_layers, "num_heads": self.num_heads,
                "num_kv_heads": self.num_kv_heads, "head_dim": self.head_dim, "intermediate_size": self.intermediate_size}

    @classmethod
    def from_dict(cls, raw: dict) -> "GogivikConfig":
        return cls(**{k: v for k, v in raw.items() if k in cls.__dataclass_fields__})

    @classmethod
    def periodic(cls, *, vocab_size: int, hidden_size: int, num_layers: int, mixers: list, ff: int, conv_taps: int = 4, logit_scale: float = 1.0,
                 norm_eps: float = 1e-5, name: str = "gogivik") -> "GogivikConfig":
        """The mixers again and again (benchmarks)."""
        return cls(vocab_size, hidden_size, [LayerSpec(mixers[i % len(mixers)], ff) for i in range(num_layers)], conv_taps, logit_scale, norm_eps, name)


def tensor_shapes(cfg: GogivikConfig) -> dict[str, tuple[int, ...]]:
    """Canonical names and shapes of a checkpoint of this design."""
    h, out = cfg.hidden_size, {}
    out["model.token_embedding.weight"] = out["model.output.weight"] = (cfg.vocab_size, h)
    out["model.output_norm.weight"] = (h,)
    for i, l in enumerate(cfg.layers):
        m, block = l.mixer, f"model.block.{i}."
        out |= {block + "attention.norm.weight": (h,), block + "attention.input_conv.weight": (h, cfg.conv_taps)}
        p = block + "attention."
        if l.kind == "latent_attention":
            out |= {p + "query_down.weight": (m.q_rank, h), p + "query_norm.weight": (m.q_rank,),
                    p + "query.weight": (m.heads * (m.dim + m.rot_dim), m.q_rank), p + "latent.weight": (m.kv_rank + m.rot_dim, h),
                    p + "latent_norm.weight": (m.kv_rank,), p + "key_up.weight": (m.heads * m.dim, m.kv_rank),
                    p + "value_up.weight": (m.heads * m.vdim, m.kv_rank), p + "sink": (m.heads,), p + "output.weight": (h, m.heads * m.vdim)}
        elif l.kind == "attention":
            out |= {p + "query.weight": (m.heads * m.dim, h), p + "key.weight": (m.kv_heads * m.dim, h), p + "value.weight": (m.kv_heads * m.vdim, h),
                    p + "query_norm.weight": (m.dim,), p + "key_norm.weight": (m.dim,), p + "output.weight": (h, m.heads * m.vdim)}
        else:
            p, inner, side = block + "linear_attention.", m.heads * m.vdim, 2 * m.groups * m.state
            out |= {p + "in.weight": (2 * inner + side + m.heads, h), p + "in_conv.weight": (inner + side, m.taps), p + "in_conv.bias": (inner + side,),
                    p + "dt_bias": (m.heads,), p + "a": (m.heads,), p + "skip": (m.heads,), p + "norm.weight": (inner,), p + "output.weight": (h, inner)}
        if l.ff:
            p = block + "mlp."
            out |= {p + "norm.weight": (h,), p + "input_conv.weight": (h, cfg.conv_taps), p + "up.weight": (l.ff, h), p + "down.weight": (h, l.ff)}
    return out


class RandomTensors(unquantized.RandomTensors):
    """Seeded random tensors of a configuration."""

    def __init__(self, cfg: GogivikConfig, device, seed: int = 0, std: float = 0.02) -> None:
        super().__init__(tensor_shapes(cfg), device, seed, std, ("query_norm.weight", "key_norm.weight", "latent_norm.weight", "linear_attention.norm.weight"))


@dataclass
class Input:
    """What stands between the stream and a sublayer."""

    norm: torch.Tensor  # [W] fp32, one added
    conv: torch.Tensor  # [taps, W] fp32


@dataclass
class LatentWeights:
    down: DenseLinear  # rows query latent | latent | rot
    q_norm: torch.Tensor  # [q_rank] fp32
    norm: torch.Tensor  # [rank] fp32
    query: DenseLinear  # rows [head][dim | rot]
    up: LatentUp
    sink: torch.Tensor  # [heads] fp32
    o_proj: DenseLinear


@dataclass
class ChunkWeights:
    qkv: DenseLinear
    q_norm: torch.Tensor  # [dk] fp32
    k_norm: torch.Tensor
    o_proj: DenseLinear


@dataclass
class StateWeights:
    proj: DenseLinear  # rows x | B | C | z | dt
    rule: ssd.Weights
    o_proj: DenseLinear
    geometry: ssd.Geometry


@dataclass
class GogivikLayer:
    input: Input
    mixer: LatentWeights | ChunkWeights | StateWeights
    mlp_input: Input | None
    up: DenseLinear | None
    down: DenseLinear | None


class GogivikWeights:
    """Weights in the layout the kernels read (widths rounded up, padding zero), on one device in one element type."""

    tp_rank, tp_size, mtp = 0, 1, None

    def __init__(self, cfg: GogivikConfig, tensors, device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``tensors``: canonical name -> checkpoint tensor (anything ``formats.dequantize`` reads, or a torch tensor)."""
        r = TensorReader(tensors, device, dtype)
        self.dtype = dtype
        w = up(cfg.hidden_size)
        self.embed = r.matrix("model.token_embedding.weight", cfg.vocab_size, w)
        self.lm_head = r.linear("model.output", up(cfg.vocab_size), w)
        self.final_norm = r.vec("model.output_norm.weight", w, offset=1.0) * cfg.logit_scale  # the logits' scale rides on the norm
        make = {"latent_attention": self._latent, "attention": self._chunked, "mamba2": self._state}
        self.layers: list[GogivikLayer] = []
        for i, l in enumerate(cfg.layers):
            p = f"model.block.{i}."
            mlp = (None, None, None)
            if l.ff:
                fp = up(l.ff)
                mlp = self._input(r, cfg, p + "mlp.", w), DenseLinear(r.matrix(p + "mlp.up.weight", fp, w), act="relu2"), r.linear(p + "mlp.down", w, fp)
            self.layers.append(GogivikLayer(self._input(r, cfg, p + "attention.", w), make[l.kind](r, cfg, l.mixer, p, w), *mlp))

    @staticmethod
    def _input(r: TensorReader, cfg: GogivikConfig, p: str, w: int) -> Input:
        return Input(r.vec(p + "norm.weight", w, offset=1.0), fit(r.get(p + "input_conv.weight").float(), w, cfg.conv_taps).T.contiguous())

    @staticmethod
    def _latent(r: TensorReader, cfg: GogivikConfig, m: LatentSpec, p: str, w: int) -> LatentWeights:
        p += "attention."
        qr, rank, rot = up(m.q_rank), up(m.kv_rank), up(m.rot_dim)
        c = r.get(p + "latent.weight").to(r.dtype)
        parts = [r.matrix(p + "query_down.weight", qr, w), fit(c[: m.kv_rank], rank, w), fit(c[m.kv_rank :], rot, w)]
        return LatentWeights(DenseLinear(torch.cat(parts).contiguous()), r.vec(p + "query_norm.weight", qr), r.vec(p + "latent_norm.weight", rank),
                             DenseLinear(latent.head_rows(r.get(p + "query.weight").to(r.dtype), m, qr).contiguous()), LatentUp.read(r, m, p),
                             r.vec(p + "sink", m.heads), DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, up(m.vdim))))

    @staticmethod
    def _chunked(r: TensorReader, cfg: GogivikConfig, m: ChunkSpec, p: str, w: int) -> ChunkWeights:
        p += "attention."
        dk, dv = up(m.dim), up(m.vdim)
        rows = [r.heads(p + n + ".weight", heads, d, dp, cfg.hidden_size, w).reshape(-1, w)
                for n, heads, d, dp in (("query", m.heads, m.dim, dk), ("key", m.kv_heads, m.dim, dk), ("value", m.kv_heads, m.vdim, dv))]
        return ChunkWeights(DenseLinear(torch.cat(rows).contiguous()), r.vec(p + "query_norm.weight", dk), r.vec(p + "key_norm.weight", dk),
                            DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, dv)))

    @staticmethod
    def _state(r: TensorReader, cfg: GogivikConfig, m: StateSpec, p: str, w: int) -> StateWeights:
        p += "linear_attention."
        n, e, inner, side = up(m.state), up(m.vdim), m.heads * m.vdim, m.groups * m.state
        geo = ssd.Geometry(m.heads, m.groups, n, e, m.vdim, m.taps, m.norm_groups, cfg.norm_eps)

        def packed(t: torch.Tensor) -> torch.Tensor:
            """Rows x | B | C, every head's and group's run padded."""
            x, b, c = t.split([inner, side, side])
            pad = lambda u, k, d, dp: fit(u.reshape(k, d, *t.shape[1:]), k, dp, *t.shape[1:]).reshape(k * dp, *t.shape[1:])
            return torch.cat([pad(x, m.heads, m.vdim, e), pad(b, m.groups, m.state, n), pad(c, m.groups, m.state, n)])
        z, xbc, dt = r.get(p + "in.weight").to(r.dtype).split([inner, inner + 2 * side, m.heads])
        z = fit(z.reshape(m.heads, m.vdim, -1), m.heads, e, w).reshape(-1, w)
        proj = torch.cat([packed(fit(xbc, xbc.shape[0], w)), z, fit(dt, up(m.heads), w)])
        taps = packed(r.get(p + "in_conv.weight").float())
        rule = ssd.Weights(taps.T.contiguous(), packed(r.get(p + "in_conv.bias").float().reshape(-1)).contiguous(), r.vec(p + "dt_bias", m.heads),
                           r.vec(p + "a", m.heads).exp(), r.vec(p + "skip", m.heads),
                           fit(r.get(p + "norm.weight").float().reshape(m.heads, m.vdim), m.heads, e).reshape(-1).contiguous())
        return StateWeights(DenseLinear(proj.contiguous()), rule, DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, e)), geo)

    def nbytes(self) -> int:
        from .hybrid import _tensor_bytes
        return _tensor_bytes([self.embed, self.lm_head, self.final_norm, self.layers])


class GogivikModel(RecurrentModel):
    def __init__(self, cfg: GogivikConfig, weights: GogivikWeights, collective=None) -> None:
        super().__init__(cfg, weights, collective)
        self.pages_of = {layer: n for n, layer in enumerate(cfg.owners())}

    def decode_splits(self, batch: int, longest: int) -> int:
        return max(super().decode_splits(batch, longest), latent.decode_splits(self.cfg.latent, batch, longest))

    def _sublayer_input(self, x, w: Input, state, step: StepBuffers, prefill: bool):
        how = dict(starts=step.q_starts, max_q=step.max_q, singles=step.num_decode) if prefill else {}
        return dense.norm_conv_out(x, w.norm, w.conv, state, step.state_slots, self.cfg.hidden_size, self.cfg.norm_eps, self.w.dtype, **how)

    # -- mixers -----------------------------------------------------------------------------------------------------
    def _latent_at(self, i: int, h, cache, step: StepBuffers, prefill: bool):
        m, w = self.cfg.layers[i].mixer, self.w.layers[i].mixer
        pages, rope = cache.layer(self.pages_of[i]).k, self._rope.get(m.rotation)
        with scope("latent.proj", h.device):
            low = latent_attn.down(w.down(h), pages, step.positions, step.slots, q_rank=up(m.q_rank), real_q_rank=m.q_rank, rank=up(m.kv_rank),
                                   rot=up(m.rot_dim), real_rank=m.kv_rank, real_rot=m.rot_dim, q_norm=w.q_norm, norm_w=w.norm, rope=rope,
                                   eps=self.cfg.norm_eps)
            q = w.query(low)
        with scope("latent.core", h.device):
            return latent.attend(self, m, w.up, q, pages, step, prefill, rope=rope, own_rows=False, sink=w.sink)

    def _chunked_at(self, i: int, h, cache, step: StepBuffers, prefill: bool):
        m, w, kv = self.cfg.layers[i].mixer, self.w.layers[i].mixer, cache.layer(self.pages_of[i])
        t, turn = h.shape[0], ValueTurn(self._rope[m.value_rotation], m.vdim)
        with scope("attn.qkv", h.device):
            qkv = w.qkv(h)
        with scope("attn.core", h.device):
            q = window_attn.qkv_finish(qkv, kv, step.positions, step.slots, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, q_norm=w.q_norm,
                                       k_norm=w.k_norm, rope=self._rope.get(m.rotation), rot=m.rot_dims, eps=self.cfg.norm_eps, turn=turn)
            how = dict(window=NO_WINDOW, chunk=m.chunk, scale=m.scale, cap=0.0)
            if h.dtype == torch.float32:
                a = window_attn.plain(q, kv, step.block_table, self._sequence_of_rows(step, t), step.positions, **how)
                return window_attn.turn_back(a, turn, step.positions).view(t, -1)
            singles = step.num_decode if prefill else t
            out = torch.empty((t, m.heads, kv.v.shape[-1]), dtype=q.dtype, device=q.device)
            if singles:
                splits = min(self.attn_splits, window_attn.decode_splits(singles, m.kv_heads, m.chunk))
                window_attn.decode(q[:singles], kv, step.block_table[:singles], step.seq_lens[:singles], turn=turn, splits=splits, out=out[:singles], **how)
            if singles < t:
                window_attn.prefill(q, kv, step.block_table[singles:], step.q_starts[singles:], step.seq_lens[singles:], step.max_q, out=out, **how)
                window_attn.turn_back(out[singles:], turn, step.positions[singles:])
            return out.view(t, -1)

    def _state_at(self, i: int, h, cache, step: StepBuffers, prefill: bool):
        w = self.w.layers[i].mixer
        with scope("ssd.proj", h.device):
            proj = w.proj(h)
        with scope("ssd.core", h.device):
            return ssd.ragged(proj, w.rule, self.state.layer((i, "state")), self.state.layer((i, "conv")), step.state_slots, w.geometry,
                              step.q_starts if prefill else None, step.max_q, step.num_decode)

    def forward(self, step: StepBuffers, cache, *, prefill: bool, logits_rows: torch.Tensor | None = None,
                gather_logits: bool = True, return_hidden: bool = False, layer_outputs: list | None = None):
        """Logits ``[rows, vocab]`` in the model's element type (all tokens, or ``logits_rows`` of them).  ``prefill``: a
        ragged batch whose first ``step.num_decode`` rows are single tokens; otherwise one token per sequence.
        ``layer_outputs`` receives a copy of the fp32 stream after every layer."""
        cfg, width = self.cfg, self.cfg.hidden_size
        x, _ = dense.embed_scaled(step.input_ids, self.w.embed, copy=False)
        run = {"latent_attention": self._latent_at, "attention": self._chunked_at, "mamba2": self._state_at}
        for i, (l, w) in enumerate(zip(cfg.layers, self.w.layers)):
            h = self._sublayer_input(x, w.input, self.state.layer((i, "input")), step, prefill)
            y = run[l.kind](i, h, cache, step, prefill)
            with scope("o_proj", x.device):
                w.mixer.o_proj(y, add_to=x)
            if w.up is not None:
                h = self._sublayer_input(x, w.mlp_input, self.state.layer((i, "mlp_input")), step, prefill)
                with scope("ffn", x.device):
                    w.down(w.up(h), add_to=x)
            if layer_outputs is not None:
                layer_outputs.append(x[:, :width].clone())
        rows = x if logits_rows is None else x.index_select(0, logits_rows.long())
        with scope("head", x.device):
            h = dense.norm_out(rows, self.w.final_norm, width, cfg.norm_eps, self.w.dtype)
            logits = self.w.lm_head(h)[:, : cfg.vocab_size]
        return (logits, x) if return_hidden else logits

"""Bufolorn: a decoder whose layers, in any order, mix by latent attention, by a delta rule with per-channel decays, or by attention
and time mixing side by side, with dense or expert feed-forwards, in bf16 or fp32.

A layer has one layer norm ``h = norm(x)`` and adds both sublayers to the fp32 stream: ``x += m (mixer(h) + ff(h))``.

* latent attention (:mod:`~mfq_b200.ops.latent_attn`): keys and values come from one normed latent per token plus one rotated key part
  shared by all heads; a sliding window; YaRN frequencies.  A layer with ``kv_from`` reads the pages of that earlier layer through
  its own expansions;
* delta rule (:mod:`~mfq_b200.ops.delta`): a matrix state per head with a decay per key channel, behind short convolutions;
* parallel: ``left_scale * attention + right_scale * time mixing``.  The attention (:mod:`~mfq_b200.ops.window_attn`) has per-head
  normalised queries and keys, a query temperature, a score cap, a learned bias by distance and a sink; the time mixing
  (:mod:`~mfq_b200.ops.gla`) reads mixes of a token and its predecessor and weighs the current token by a bonus;
* feed-forward: ``W_down (max(gate, 0) * up)``, or routed experts (:mod:`~mfq_b200.ops.dense_moe`) with sigmoid scores, a choice
  correction and a shared expert.

Layers may differ in kind and in every size and constant.  Runs on a CUDA device only; batches are ragged.
"""

from __future__ import annotations

import math
from dataclasses import asdict, dataclass, field

import torch

from ..ops import delta, dense, dense_moe, gla, window_attn
from ..ops.dense import DenseLinear, up
from ..ops.window_attn import NO_WINDOW, DistanceBias
from ..utils.profiler import scope
from . import latent, unquantized
from .latent import LatentUp
from .llama import StepBuffers
from .rope_scaling import YarnScaling
from .unquantized import RecurrentModel, TensorReader, fit


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int  # unrotated query / key channels per head
    rot_dim: int  # rotated ones
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float = 1e4
    rot_scaling: YarnScaling | None = None
    window: int = NO_WINDOW
    kv_from: int | None = None  # the layer whose latents this one reads

    @property
    def rotation(self) -> tuple:
        return self.rot_base, self.rot_dim, self.rot_scaling

    @property
    def row(self) -> int:
        """Stored width of a token's row of the cache."""
        return up(self.kv_rank) + up(self.rot_dim)


@dataclass(frozen=True)
class BiasedSpec:
    """The attention of a parallel layer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float  # 0: none
    bias_max: float
    temp_coef: float = 0.0
    temp_every: int = 1
    buckets: int = 0  # rows of the distance table; 0: what the checkpoint's tensor has


@dataclass(frozen=True)
class TimeMixSpec:
    heads: int
    dim: int
    rank: int = 0  # of the decay projection; 0: what the checkpoint's tensors have


@dataclass(frozen=True)
class ParallelSpec:
    left: BiasedSpec
    right: TimeMixSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    rank_a: int = 0  # of the decay and gate projections; 0: what the checkpoint's tensors have
    rank_g: int = 0


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    scale: float
    ff: int
    shared: int = 0  # width of the shared expert; 0: none


MIXERS = {"latent_attention": LatentSpec, "parallel": ParallelSpec, "channel_delta": DeltaSpec}


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec | ParallelSpec | DeltaSpec
    mlp: DenseSpec | ExpertsSpec | None = None

    @property
    def kind(self) -> str:
        return next(k for k, c in MIXERS.items() if isinstance(self.mixer, c))

    @classmethod
    def from_dict(cls, raw: dict) -> "LayerSpec":
        m, mlp = dict(raw["mixer"]), raw.get("mlp")
        if "left" in m:
            mixer = ParallelSpec(BiasedSpec(**m["left"]), TimeMixSpec(**m["right"]), m["left_scale"], m["right_scale"])
        elif "taps" in m:
            mixer = DeltaSpec(**m)
        else:
            mixer = LatentSpec(**{**m, "rot_scaling": YarnScaling.from_dict(m.get("rot_scaling"))})
        if mlp is not None:
            mlp = ExpertsSpec(**mlp) if "experts" in mlp else DenseSpec(**mlp)
        return cls(mixer, mlp)


def _yarn(raw: dict | None) -> YarnScaling | None:
    if not raw:
        return None
    factor = float(raw["factor"])
    return YarnScaling(factor, raw["original"], float(raw["fast"]), float(raw["slow"]), attention_factor=0.1 * math.log(factor) + 1.0)


@dataclass
class BufolornConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    norm_eps: float = 1e-5
    name: str = "bufolorn"

    def __post_init__(self):
        self.layers = [l if isinstance(l, LayerSpec) else LayerSpec.from_dict(l) for l in self.layers]
        for i, l in enumerate(self.layers):
            try:
                self._check(i, l)
            except ValueError as exc:
                raise ValueError(f"layer {i}: {exc}") from None

    def _check(self, i: int, l: LayerSpec) -> None:
        m = l.mixer
        if l.kind == "latent_attention":
            latent.check_sizes(m)
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, LatentSpec) or src.kv_from is not None:
                    raise ValueError(f"layer {m.kv_from} has no latents to read")
                if (src.kv_rank, src.rotation) != (m.kv_rank, m.rotation):
                    raise ValueError(f"its latents differ from those of layer {m.kv_from}")
        elif l.kind == "parallel":
            a, t = m.left, m.right
            if min(a.heads, a.kv_heads, a.dim, a.vdim) < 1 or a.heads % a.kv_heads or a.heads // a.kv_heads > 128 or not a.scale > 0:
                raise ValueError(f"unsupported attention {a}")
            if max(a.dim, a.vdim) > window_attn.MAX_HEAD or a.softcap < 0 or a.temp_every < 1:
                raise ValueError(f"unsupported attention {a}")
            if min(t.heads, t.dim) < 1 or up(t.dim) > 1024:
                raise ValueError(f"unsupported time mixing {t}")
        else:
            if min(m.heads, m.kv_heads, m.dim, m.vdim) < 1 or m.heads % m.kv_heads or not 1 <= m.taps <= 8:
                raise ValueError(f"unsupported delta rule {m}")
            if not delta.column_split(1, m.heads, up(m.dim), up(m.vdim)):
                raise ValueError(f"a state of {m.dim} x {m.vdim} per head is not supported")
        if isinstance(l.mlp, ExpertsSpec) and not (1 <= l.mlp.top <= min(16, l.mlp.experts) and l.mlp.experts <= 512 and l.mlp.ff > 0):
            raise ValueError(f"unsupported experts {l.mlp}")
        if isinstance(l.mlp, DenseSpec) and l.mlp.ff < 1:
            raise ValueError(f"unsupported feed-forward {l.mlp}")

    # -- what other parts of the framework ask a configuration for ------------------------------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def _of(self, kind: str) -> list:
        return [l.mixer for l in self.layers if l.kind == kind]

    @property
    def attention(self) -> list[BiasedSpec]:
        return [m.left for m in self._of("parallel")]

    @property
    def latent(self) -> list[LatentSpec]:
        return self._of("latent_attention")

    @property
    def num_heads(self) -> int:
        return max([m.heads for m in self.latent + self.attention + self._of("channel_delta")])

    @property
    def num_kv_heads(self) -> int:
        return max([m.kv_heads for m in self.attention], default=1)

    @property
    def head_dim(self) -> int:
        return max(max(m.dim, m.vdim) for m in self.latent + self.attention + self._of("channel_delta"))

    @property
    def intermediate_size(self) -> int:
        return max((l.mlp.ff for l in self.layers if l.mlp is not None), default=0)

    def owners(self) -> list[int]:
        """Layers with pages of their own, in order: place in the cache -> layer."""
        return [i for i, l in enumerate(self.layers) if l.kind == "parallel" or (l.kind == "latent_attention" and l.mixer.kv_from is None)]

    def kv_shapes(self) -> list[tuple[int, int, int]]:
        """Per layer with pages: (KV heads, stored key width, stored value width).  A latent row is the key; its values are part of it."""
        out = []
        for m in (self.layers[i].mixer for i in self.owners()):
            out.append((1, m.row, 0) if isinstance(m, LatentSpec) else (m.left.kv_heads, up(m.left.dim), up(m.left.vdim)))
        return out

    def kv_token_bytes(self, element_bytes: int) -> int:
        return sum(g * (dk + dv) for g, dk, dv in self.kv_shapes()) * element_bytes

    def state_shapes(self) -> dict[tuple[int, str], tuple[int, ...]]:
        """(layer, part) -> shape of a sequence's fp32 state."""
        out = {}
        for i, l in enumerate(self.layers):
            m = l.mixer
            if l.kind == "channel_delta":
                dk, dv = up(m.dim), up(m.vdim)
                out[i, "state"] = (m.heads, dk, dv)
                out[i, "conv"] = (m.taps - 1, 2 * m.kv_heads * dk + m.heads * dv)
            elif l.kind == "parallel":
                d = up(m.right.dim)
                out[i, "state"] = (m.right.heads, d, d)
                out[i, "last"] = (up(self.hidden_size),)
        return out

    def state_bytes(self) -> int:
        return sum(4 * math.prod(s) for s in self.state_shapes().values())

    def rotations(self) -> set[tuple]:
        return {m.rotation for m in self.latent}

    def key_spans(self) -> list[tuple[int, int, int]]:
        """Per attention layer over keys of its own: (KV heads, window, kept first keys)."""
        return [(m.kv_heads, NO_WINDOW, 0) for m in self.attention]

    @property
    def attention_layers(self) -> int:
        return len(self.latent) + len(self.attention)

    def param_count(self) -> int:
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    # -- forms ----------------------------------------------------------------------------------------------------------
    @classmethod
    def from_source(cls, src: dict) -> "BufolornConfig":
        """The model's own ``config.json``."""
        ints = lambda m, *names: {n: int(m[n]) for n in names}
        layers = []
        for i, entry in enumerate(src["layers"]):
            m, mlp, kind = entry["mixer"], entry.get("mlp"), entry.get("type")
            if kind == "latent_attention":
                rot = m["rot"]
                if int(rot["dims"]) != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: {rot['dims']} rotated channels of a rotated part of {m['rot_dim']}")
                mixer = LatentSpec(**ints(m, "heads", "dim", "rot_dim", "vdim", "kv_rank"), scale=float(m["scale"]), rot_base=float(rot["base"]),
                                   rot_scaling=_yarn(rot.get("scaling")), window=min(int((m.get("mask") or {}).get("size") or NO_WINDOW), NO_WINDOW),
                                   kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
            elif kind == "parallel":
                a, temp = m["left"], m["left"].get("q_temp") or {"coef": 0.0, "every": 1}
                mixer = ParallelSpec(BiasedSpec(**ints(a, "heads", "kv_heads", "dim", "vdim"), scale=float(a["scale"]),
                                                softcap=float(a.get("softcap") or 0.0), bias_max=float(a["bias_max"]),
                                                temp_coef=float(temp["coef"]), temp_every=int(temp["every"])),
                                     TimeMixSpec(**ints(m["right"], "heads", "dim")), float(m["left_scale"]), float(m["right_scale"]))
            elif kind == "channel_delta":
                mixer = DeltaSpec(**ints(m, "heads", "kv_heads", "dim", "vdim"), taps=int(m["conv"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            if mlp is None:
                ff = None
            elif mlp.get("kind") == "dense":
                ff = DenseSpec(int(mlp["ff"]))
            elif mlp.get("kind") == "moe":
                r = mlp["router"]
                ff = ExpertsSpec(int(r["experts"]), int(r["top"]), float(r["scale"]), int(mlp["expert"]["ff"]),
                                 int((mlp.get("shared") or {}).get("ff", 0)))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            layers.append(LayerSpec(mixer, ff))
        return cls(vocab_size=int(src["vocab"]), hidden_size=int(src["width"]), layers=layers, embed_scale=float(src["embedding"]["scale"]),
                   residual_mult=float(src["residual_mult"]), norm_eps=float(src["norm"]["eps"]))

    def to_dict(self) -> dict:
        """The form checkpoints carry: this class's fields plus the summary keys other tools read."""
        return {**asdict(self), "family": "bufolorn", "num_layers": self.num_layers, "num_heads": self.num_heads,
                "num_kv_heads": self.num_kv_heads, "head_dim": self.head_dim, "intermediate_size": self.intermediate_size}

    @classmethod
    def from_dict(cls, raw: dict) -> "BufolornConfig":
        return cls(**{k: v for k, v in raw.items() if k in cls.__dataclass_fields__})

    @classmethod
    def periodic(cls, *, vocab_size: int, hidden_size: int, num_layers: int, latent: LatentSpec, delta_rule: DeltaSpec, parallel: ParallelSpec,
                 mlp: list, embed_scale: float = 1.0, residual_mult: float = 1.0, norm_eps: float = 1e-5, name: str = "bufolorn") -> "BufolornConfig":
        """Latent, delta rule, parallel, and latent attention on the latents of three layers before, again and again; the feed-forwards
        go round in a period of their own (benchmarks)."""
        layers = []
        for i in range(num_layers):
            again = LatentSpec(**{**vars(latent), "kv_from": i - 3})
            layers.append(LayerSpec((latent, delta_rule, parallel, again)[i % 4], mlp[i % len(mlp)]))
        return cls(vocab_size, hidden_size, layers, embed_scale, residual_mult, norm_eps, name)


def tensor_shapes(cfg: BufolornConfig) -> dict[str, tuple[int, ...]]:
    """Canonical names and shapes of a checkpoint of this design (ranks and distance tables as far as the configuration knows them)."""
    h, out = cfg.hidden_size, {}
    out["model.token_embedding.weight"] = out["model.output.weight"] = (cfg.vocab_size, h)
    out["model.output_norm.weight"] = out["model.output_norm.bias"] = (h,)
    for i, l in enumerate(cfg.layers):
        m, block = l.mixer, f"model.block.{i}."
        out[block + "norm.weight"] = out[block + "norm.bias"] = (h,)
        if l.kind == "latent_attention":
            p = block + "attention."
            out |= {p + "query.weight": (m.heads * (m.dim + m.rot_dim), h), p + "output.weight": (h, m.heads * m.vdim),
                    p + "key_up.weight": (m.heads * m.dim, m.kv_rank), p + "value_up.weight": (m.heads * m.vdim, m.kv_rank)}
            if m.kv_from is None:
                out |= {p + "latent.weight": (m.kv_rank + m.rot_dim, h), p + "latent_norm.weight": (m.kv_rank,)}
        elif l.kind == "parallel":
            a, t, p = m.left, m.right, block + "attention."
            for n, rows in (("query", a.heads * a.dim), ("key", a.kv_heads * a.dim), ("value", a.kv_heads * a.vdim)):
                out |= {p + n + ".weight": (rows, h), p + n + ".bias": (rows,)}
            out |= {p + "output.weight": (h, a.heads * a.vdim), p + "output.bias": (h,), p + "distance.bias": (a.buckets, a.heads),
                    p + "sink": (a.heads,)}
            p, w = block + "time_mixing.", t.heads * t.dim
            out |= {p + f"{n}_mix": (h,) for n in ("receptance", "key", "value", "gate", "decay")}
            out |= {p + n + ".weight": (w, h) for n in ("receptance", "key", "value", "gate")}
            out |= {p + "decay_a.weight": (t.rank, h), p + "decay_b.weight": (w, t.rank), p + "decay_b.bias": (w,), p + "bonus": (t.heads, t.dim),
                    p + "norm.weight": (w,), p + "output.weight": (h, w)}
        else:
            p = block + "linear_attention."
            for n, rows in (("query", m.kv_heads * m.dim), ("key", m.kv_heads * m.dim), ("value", m.heads * m.vdim)):
                out |= {p + n + ".weight": (rows, h), p + n + "_conv.weight": (rows, m.taps)}
            out |= {p + "beta.weight": (m.heads, h), p + "a": (m.heads,), p + "dt_bias": (m.heads * m.dim,), p + "norm.weight": (m.vdim,),
                    p + "decay_a.weight": (m.rank_a, h), p + "decay_b.weight": (m.heads * m.dim, m.rank_a),
                    p + "gate_a.weight": (m.rank_g, h), p + "gate_b.weight": (m.heads * m.vdim, m.rank_g),
                    p + "output.weight": (h, m.heads * m.vdim)}
        unit = lambda p, f: {p + "gate.weight": (f, h), p + "up.weight": (f, h), p + "down.weight": (h, f)}
        if isinstance(l.mlp, DenseSpec):
            out |= unit(block + "mlp.", l.mlp.ff)
        elif l.mlp is not None:
            e = l.mlp.experts
            out |= {n: (e, *s) for n, s in unit(block + "mlp.experts.", l.mlp.ff).items()}
            out |= {block + "mlp.router.weight": (e, h), block + "mlp.router.bias": (e,)}
            if l.mlp.shared:
                out |= unit(block + "mlp.shared_expert.", l.mlp.shared)
    return out


class RandomTensors(unquantized.RandomTensors):
    """Seeded random tensors of a configuration (whose layers give their ranks and distance tables)."""

    def __init__(self, cfg: BufolornConfig, device, seed: int = 0, std: float = 0.02) -> None:
        super().__init__(tensor_shapes(cfg), device, seed, std, ("norm.weight",))


@dataclass
class LatentWeights:
    proj: DenseLinear  # rows [head][dim | rot], then [latent | rot] in a layer with pages of its own
    norm: torch.Tensor | None  # [rank] fp32
    up: LatentUp
    o_proj: DenseLinear


@dataclass
class ParallelWeights:
    qkv: DenseLinear
    ones: torch.Tensor  # [dk]: the norm of q and k has no weight
    bias: DistanceBias
    sink: torch.Tensor  # [heads] fp32
    attn_out: DenseLinear
    mu: torch.Tensor  # [5, W] fp32: r, k, v, g, w
    rkvg: DenseLinear  # a matrix per stream
    decay_a: DenseLinear
    decay_b: torch.Tensor  # [heads * d, rank]
    decay_bias: torch.Tensor  # [heads * d] fp32
    bonus: torch.Tensor  # [heads * d] fp32
    norm: torch.Tensor  # [heads, d] fp32
    mix_out: DenseLinear
    geometry: gla.Geometry


@dataclass
class DeltaWeights:
    proj: DenseLinear  # rows q | k | v | b | a | g
    rule: delta.Weights
    o_proj: DenseLinear
    geometry: delta.Geometry


@dataclass
class DenseFf:
    gate_up: DenseLinear
    down: DenseLinear


@dataclass
class ExpertsFf:
    router: dense_moe.Router
    bank: dense_moe.ExpertBank
    shared: DenseFf | None


@dataclass
class BufolornLayer:
    norm: torch.Tensor  # [W] fp32
    norm_bias: torch.Tensor
    mixer: LatentWeights | ParallelWeights | DeltaWeights
    mlp: DenseFf | ExpertsFf | None


class BufolornWeights:
    """Weights in the layout the kernels read (widths rounded up, padding zero), on one device in one element type."""

    tp_rank, tp_size, mtp = 0, 1, None

    def __init__(self, cfg: BufolornConfig, tensors, device, dtype: torch.dtype = torch.bfloat16) -> None:
        """``tensors``: canonical name -> checkpoint tensor (anything ``formats.dequantize`` reads, or a torch tensor)."""
        r = TensorReader(tensors, device, dtype)
        self.dtype = dtype
        w = up(cfg.hidden_size)
        self.embed = r.matrix("model.token_embedding.weight", cfg.vocab_size, w)
        self.lm_head = r.linear("model.output", up(cfg.vocab_size), w)
        self.final_norm, self.final_bias = r.vec("model.output_norm.weight", w), r.vec("model.output_norm.bias", w)
        make = {"latent_attention": self._latent, "parallel": self._parallel, "channel_delta": self._delta}
        self.layers: list[BufolornLayer] = []
        for i, l in enumerate(cfg.layers):
            p = f"model.block.{i}."
            mlp = None
            if isinstance(l.mlp, DenseSpec):
                mlp = self._unit(r, p + "mlp.", l.mlp.ff, w, "relu")
            elif l.mlp is not None:
                mlp = self._experts(r, l.mlp, p + "mlp.", w)
            self.layers.append(BufolornLayer(r.vec(p + "norm.weight", w), r.vec(p + "norm.bias", w), make[l.kind](r, cfg, l.mixer, p, w), mlp))

    @staticmethod
    def _latent(r: TensorReader, cfg: BufolornConfig, m: LatentSpec, p: str, w: int) -> LatentWeights:
        p += "attention."
        rot, rank = up(m.rot_dim), up(m.kv_rank)
        parts, norm = [latent.head_rows(r.get(p + "query.weight").to(r.dtype), m, w)], None
        if m.kv_from is None:
            c = r.get(p + "latent.weight").to(r.dtype)
            parts += [fit(c[: m.kv_rank], rank, w), fit(c[m.kv_rank :], rot, w)]
            norm = r.vec(p + "latent_norm.weight", rank)
        return LatentWeights(DenseLinear(torch.cat(parts).contiguous()), norm, LatentUp.read(r, m, p),
                             DenseLinear(r.from_heads(p + "output.weight", cfg.hidden_size, w, m.heads, m.vdim, up(m.vdim))))

    @staticmethod
    def _parallel(r: TensorReader, cfg: BufolornConfig, m: ParallelSpec, p: str, w: int) -> ParallelWeights:
        a, t, width = m.left, m.right, cfg.hidden_size
        q, dk, dv = p + "attention.", up(a.dim), up(a.vdim)
        rows, biases = [], []
        for name, heads, d, dp in (("query", a.heads, a.dim, dk), ("key", a.kv_heads, a.dim, dk), ("value", a.kv_heads, a.vdim, dv)):
            rows.append(r.heads(q + name + ".weight", heads, d, dp, width, w).reshape(-1, w))
            biases.append(fit(r.get(q + name + ".bias").float().reshape(heads, d), heads, dp).reshape(-1))
        table = r.get(q + "distance.bias").float()
        buckets = table.shape[0]
        if buckets < 2 or not a.bias_max > buckets // 2 or (a.buckets and a.buckets != buckets):
            raise ValueError(f"{q}distance.bias: a table of {buckets} rows does not reach {a.bias_max:g}")
        bias = DistanceBias.from_table(table[torch.tensor(window_attn.log_buckets(buckets, a.bias_max), device=table.device)].T)
        s, d = p + "time_mixing.", up(t.dim)
        streams = ("receptance", "key", "value", "gate")
        rank = r.get(s + "decay_a.weight").shape[0]
        if t.rank and t.rank != rank:
            raise ValueError(f"{s}decay_a has rank {rank}, the configuration says {t.rank}")
        geo = gla.Geometry(t.heads, d, d, t.dim, t.dim, up(rank), 1.0, cfg.norm_eps, decay="exp", scaled=False)
        per_head = lambda name: fit(r.get(s + name).float().reshape(t.heads, t.dim), t.heads, d).contiguous()
        return ParallelWeights(
            DenseLinear(torch.cat(rows).contiguous(), torch.cat(biases).contiguous()), fit(torch.ones(a.dim, device=r.device), dk).contiguous(), bias,
            r.vec(q + "sink", a.heads), DenseLinear(r.from_heads(q + "output.weight", width, w, a.heads, a.vdim, dv), r.vec(q + "output.bias", w)),
            torch.stack([r.vec(s + n + "_mix", w) for n in (*streams, "decay")]),
            DenseLinear(torch.cat([r.heads(s + n + ".weight", t.heads, t.dim, d, width, w).reshape(-1, w) for n in streams]).contiguous(), groups=4),
            DenseLinear(r.matrix(s + "decay_a.weight", geo.rank, w)),
            r.heads(s + "decay_b.weight", t.heads, t.dim, d, rank, geo.rank).reshape(-1, geo.rank).contiguous(), per_head("decay_b.bias").reshape(-1),
            per_head("bonus").reshape(-1), per_head("norm.weight"),
            DenseLinear(r.from_heads(s + "output.weight", width, w, t.heads, t.dim, d)), geo)

    @staticmethod
    def _delta(r: TensorReader, cfg: BufolornConfig, m: DeltaSpec, p: str, w: int) -> DeltaWeights:
        p += "linear_attention."
        dk, dv, width = up(m.dim), up(m.vdim), cfg.hidden_size
        rank_a, rank_g = (r.get(p + n + ".weight").shape[0] for n in ("decay_a", "gate_a"))
        if (m.rank_a and m.rank_a != rank_a) or (m.rank_g and m.rank_g != rank_g):
            raise ValueError(f"{p}decay_a / gate_a have ranks {rank_a} / {rank_g}, the configuration says {m.rank_a} / {m.rank_g}")
        geo = delta.Geometry(m.heads, m.kv_heads, dk, dv, m.dim, m.vdim, up(rank_a), up(rank_g), m.taps, cfg.norm_eps)
        rows, taps = [], []
        for n, heads, d, dp in (("query", m.kv_heads, m.dim, dk), ("key", m.kv_heads, m.dim, dk), ("value", m.heads, m.vdim, dv)):
            rows.append(r.heads(p + n + ".weight", heads, d, dp, width, w).reshape(-1, w))
            taps.append(fit(r.get(p + n + "_conv.weight").float().reshape(heads, d, m.taps), heads, dp, m.taps).reshape(-1, m.taps))
        rows += [r.matrix(p + "beta.weight", geo.b_cols, w), r.matrix(p + "decay_a.weight", geo.rank_a, w), r.matrix(p + "gate_a.weight", geo.rank_g, w)]
        rule = delta.Weights(torch.cat(taps).T.contiguous(), r.heads(p + "decay_b.weight", m.heads, m.dim, dk, rank_a, geo.rank_a).reshape(-1, geo.rank_a).contiguous(),
                             fit(r.get(p + "dt_bias").float().reshape(m.heads, m.dim), m.heads, dk).reshape(-1).contiguous(),
                             r.vec(p + "a", m.heads).exp(),
                             DenseLinear(r.heads(p + "gate_b.weight", m.heads, m.vdim, dv, rank_g, geo.rank_g).reshape(-1, geo.rank_g).contiguous()),
                             r.vec(p + "norm.weight", dv))
        return DeltaWeights(DenseLinear(torch.cat(rows).contiguous()), rule, DenseLinear(r.from_heads(p + "output.weight", width, w, m.heads, m.vdim, dv)), geo)

    @staticmethod
    def _unit(r: TensorReader, p: str, ff: int, w: int, act: str) -> DenseFf:
        fp = up(ff, 8)
        return DenseFf(r.glu(p, fp, w, act), r.linear(p + "down", w, fp))

    @staticmethod
    def _experts(r: TensorReader, m: ExpertsSpec, p: str, w: int) -> ExpertsFf:
        fp, e = up(m.ff, 8), m.experts
        gate, up_, down = (r.get(p + f"experts.{n}.weight").to(r.dtype) for n in ("gate", "up", "down"))
        both = torch.cat([dense.interleave_glu(fit(gate[i], fp, w), fit(up_[i], fp, w)) for i in range(e)]).contiguous()
        bank = dense_moe.ExpertBank(e, both, fit(down, e, w, fp).reshape(-1, fp).contiguous())
        router = dense_moe.Router(DenseLinear(r.matrix(p + "router.weight", up(e), w)), r.vec(p + "router.bias", e), e, m.top, m.scale)
        shared = BufolornWeights._unit(r, p + "shared_expert.", m.shared, w, "silu") if m.shared else None
        return ExpertsFf(router, bank, shared)

    def nbytes(self) -> int:
        from .hybrid import _tensor_bytes
        return _tensor_bytes([self.embed, self.lm_head, self.final_norm, self.layers])


class BufolornModel(RecurrentModel):
    def __init__(self, cfg: BufolornConfig, weights: BufolornWeights, collective=None) -> None:
        super().__init__(cfg, weights, collective)
        place = {layer: n for n, layer in enumerate(cfg.owners())}
        self.pages_of = [place.get(getattr(l.mixer, "kv_from", None) if getattr(l.mixer, "kv_from", None) is not None else i)
                         for i, l in enumerate(cfg.layers)]

    def decode_splits(self, batch: int, longest: int) -> int:
        return max(super().decode_splits(batch, longest), latent.decode_splits(self.cfg.latent, batch, longest))

    # -- mixers -----------------------------------------------------------------------------------------------------
    def _latent_at(self, i: int, h, x, cache, step: StepBuffers, prefill: bool) -> None:
        m, w = self.cfg.layers[i].mixer, self.w.layers[i].mixer
        with scope("latent.proj", x.device):
            proj = w.proj(h)
        with scope("latent.core", x.device):
            y = latent.attend(self, m, w.up, proj, cache.layer(self.pages_of[i]).k, step, prefill, rope=self._rope.get(m.rotation),
                              own_rows=m.kv_from is None, norm=w.norm)
        with scope("latent.o_proj", x.device):
            w.o_proj(y, add_to=x, scale=self.cfg.residual_mult)

    def _biased_attention(self, a: BiasedSpec, w: ParallelWeights, h, kv, step: StepBuffers, prefill: bool):
        t = h.shape[0]
        how = dict(window=NO_WINDOW, scale=a.scale, cap=a.softcap, bias=w.bias, sink=w.sink)
        q = window_attn.qkv_finish(w.qkv(h), kv, step.positions, step.slots, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, q_norm=w.ones,
                                   k_norm=w.ones, rope=None, rot=0, eps=self.cfg.norm_eps, temperature=(a.temp_coef, a.temp_every))
        if h.dtype == torch.float32:
            return window_attn.plain(q, kv, step.block_table, self._sequence_of_rows(step, t), step.positions, **how).view(t, -1)
        singles = step.num_decode if prefill else t
        out = torch.empty((t, a.heads, kv.v.shape[-1]), dtype=q.dtype, device=q.device)
        if singles:
            window_attn.decode(q[:singles], kv, step.block_table[:singles], step.seq_lens[:singles],
                               splits=min(self.attn_splits, window_attn.decode_splits(singles, a.kv_heads, NO_WINDOW)), out=out[:singles], **how)
        if prefill and singles < step.seq_lens.numel():
            window_attn.prefill(q, kv, step.block_table[singles:], step.q_starts[singles:], step.seq_lens[singles:], step.max_q, out=out, **how)
        return out.view(t, -1)

    def _time_mixing(self, i: int, w: ParallelWeights, h, step: StepBuffers, prefill: bool):
        geo, width = w.geometry, h.shape[1]
        mixes = gla.token_shift(h, w.mu, self.state.layer((i, "last")), step.state_slots, step.q_starts if prefill else None,
                                step.tok_seq if prefill else None)
        proj = torch.empty((h.shape[0], geo.width), dtype=h.dtype, device=h.device)
        streams = 4 * geo.heads * geo.dk
        w.rkvg(mixes[:, : 4 * width], out=proj[:, :streams])
        w.decay_a(mixes[:, 4 * width :], softcap=1.0, out=proj[:, streams:])  # cap 1: tanh
        args = (proj, w.decay_b, w.decay_bias, w.norm, self.state.layer((i, "state")), step.state_slots, geo)
        if prefill:
            return gla.ragged(*args, step.q_starts, step.max_q, step.num_decode, bonus=w.bonus)
        return gla.recurrent(*args, bonus=w.bonus)

    def _parallel_at(self, i: int, h, x, cache, step: StepBuffers, prefill: bool) -> None:
        m, w, mult = self.cfg.layers[i].mixer, self.w.layers[i].mixer, self.cfg.residual_mult
        with scope("parallel.attn", x.device):
            w.attn_out(self._biased_attention(m.left, w, h, cache.layer(self.pages_of[i]), step, prefill), add_to=x, scale=mult * m.left_scale)
        with scope("parallel.mix", x.device):
            w.mix_out(self._time_mixing(i, w, h, step, prefill), add_to=x, scale=mult * m.right_scale)

    def _delta_at(self, i: int, h, x, cache, step: StepBuffers, prefill: bool) -> None:
        w = self.w.layers[i].mixer
        with scope("delta.proj", x.device):
            proj = w.proj(h)
        with scope("delta.core", x.device):
            y = delta.ragged(proj, w.rule, self.state.layer((i, "state")), self.state.layer((i, "conv")), step.state_slots, w.geometry,
                             step.q_starts if prefill else None, step.max_q, step.num_decode)
        with scope("delta.o_proj", x.device):
            w.o_proj(y, add_to=x, scale=self.cfg.residual_mult)

    def _feed_forward(self, w: DenseFf | ExpertsFf, h, x) -> None:
        mult = self.cfg.residual_mult
        if isinstance(w, ExpertsFf):
            with scope("moe", x.device):
                ids, weight = w.router(h)
                dense_moe.add_experts(h, ids, weight, w.bank, x, mult)
            w = w.shared
        if w is not None:
            with scope("ffn", x.device):
                w.down(w.gate_up(h), add_to=x, scale=mult)

    def forward(self, step: StepBuffers, cache, *, prefill: bool, logits_rows: torch.Tensor | None = None,
                gather_logits: bool = True, return_hidden: bool = False, layer_outputs: list | None = None):
        """Logits ``[rows, vocab]`` in the model's element type (all tokens, or ``logits_rows`` of them).  ``prefill``: a
        ragged batch whose first ``step.num_decode`` rows are single tokens; otherwise one token per sequence.
        ``layer_outputs`` receives a copy of the fp32 stream after every layer."""
        cfg, width = self.cfg, self.cfg.hidden_size
        x, _ = dense.embed_scaled(step.input_ids, self.w.embed, cfg.embed_scale, copy=False)
        run = {"latent_attention": self._latent_at, "parallel": self._parallel_at, "channel_delta": self._delta_at}
        for i, (l, w) in enumerate(zip(cfg.layers, self.w.layers)):
            h = dense.layer_norm_out(x, w.norm, w.norm_bias, width, cfg.norm_eps, self.w.dtype)
            run[l.kind](i, h, x, cache, step, prefill)
            if w.mlp is not None:
                self._feed_forward(w.mlp, h, x)
            if layer_outputs is not None:
                layer_outputs.append(x[:, :width].clone())
        rows = x if logits_rows is None else x.index_select(0, logits_rows.long())
        with scope("head", x.device):
            h = dense.layer_norm_out(rows, self.w.final_norm, self.w.final_bias, width, cfg.norm_eps, self.w.dtype)
            logits = self.w.lm_head(h)[:, : cfg.vocab_size]
        return (logits, x) if return_hidden else logits

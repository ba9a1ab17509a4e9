"""Model families: which configuration, weights and model class serve a checkpoint.

:func:`find` picks the family from the checkpoint's canonical configuration (the keyword dict of
:func:`~mfq_b200.architectures.config_from_hf` or of ``model_config.json``); ``Family.build`` turns that configuration and the
checkpoint's tensors into ``(config, weights, model)``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(ValueError):
    """The family has no kernels for the requested element type."""


@dataclass
class LoadOptions:
    """What :func:`~mfq_b200.checkpoint.load_engine` was asked for, as far as a family's weights or model depend on it."""

    device: object = "cuda"
    dtype: str = "auto"  # element type of weights and activations; "auto": what the family serves in
    native_4bit: bool = False
    expert_slots: int | None = None
    tp_rank: int = 0
    tp_size: int = 1
    lp_rank: int = 0
    lp_size: int = 1
    layer_split: object = None
    collective: object = None


@dataclass(frozen=True)
class Family:
    name: str
    matches: Callable[[dict], bool]
    build: Callable  # (raw config, tensors, LoadOptions) -> (config, weights, model)
    dtypes: tuple[str, ...] = ("auto",)
    kernels: tuple[str, ...] = ("kernels",)  # libraries of ops.build its forward pass needs

    def check_dtype(self, dtype: str) -> None:
        if dtype not in self.dtypes:
            raise UnsupportedDtype(f"models of the {self.name} family do not run in {dtype} (available: {', '.join(self.dtypes)})")


def _unquantized(name: str, config: str, weights: str, model: str):
    """Builder of a family of the unquantized path, from the classes in ``models/<name>.py``."""
    def build(raw: dict, store, o: LoadOptions):
        from importlib import import_module
        module = import_module(f"{__package__}.{name}")
        if o.tp_size != 1 or o.lp_size != 1:
            raise NotImplementedError(f"{name} checkpoints load on a single rank")
        if raw.get("rope_scaling"):
            raise ValueError("this family has no rotary context extension")
        cfg = getattr(module, config).from_dict(raw)
        w = getattr(module, weights)(cfg, store, o.device, DTYPES["bfloat16" if o.dtype == "auto" else o.dtype])
        return cfg, w, getattr(module, model)(cfg, w, collective=o.collective)
    return Family(name, lambda raw: raw.get("family") == name, build, ("auto", "bfloat16", "float32"), ("dense",))


def _build_mla(raw: dict, store, o: LoadOptions):
    from .mla import MlaConfig, MlaModel, mla_weights_from_tensors
    if o.tp_size != 1:
        raise NotImplementedError("latent-attention checkpoints load on a single rank")
    cfg = MlaConfig(**{k: v for k, v in raw.items() if k in MlaConfig.__dataclass_fields__})
    weights = mla_weights_from_tensors(cfg, store, o.device)
    return cfg, weights, MlaModel(cfg, weights)


def _build_moe_decoder(raw: dict, store, o: LoadOptions):
    from .moe_decoder import MoeDecoderConfig, MoeDecoderModel, MoeWeights
    cfg = MoeDecoderConfig(**{k: v for k, v in raw.items() if k in MoeDecoderConfig.__dataclass_fields__})
    weights = MoeWeights.from_tensors(cfg, store, o.device, o.tp_rank, o.tp_size, expert_slots=o.expert_slots,
                                      native_4bit=o.native_4bit, lp_rank=o.lp_rank, lp_size=o.lp_size, layer_split=o.layer_split)
    return cfg, weights, MoeDecoderModel(cfg, weights, collective=o.collective)


FAMILIES = (
    _unquantized("tepetar", "TepetarConfig", "TepetarWeights", "TepetarModel"),
    _unquantized("kamedra", "KamedraConfig", "KamedraWeights", "KamedraModel"),
    _unquantized("bufolorn", "BufolornConfig", "BufolornWeights", "BufolornModel"),
    _unquantized("gogivik", "GogivikConfig", "GogivikWeights", "GogivikModel"),
    Family("latent attention", lambda raw: bool(raw.get("kv_lora_rank")), _build_mla),
    Family("decoder", lambda raw: True, _build_moe_decoder),  # dense and mixture-of-experts decoders
)


def find(raw: dict) -> Family:
    return next(f for f in FAMILIES if f.matches(raw))

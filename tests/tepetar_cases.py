"""Small Tepetar checkpoints for the tests: configurations, seeded weights, and the directory form an engine loads."""

from __future__ import annotations

import json
import struct

import numpy as np
import torch


def layer(heads=6, kv_heads=2, dim=32, vdim=24, window=40, rot=24, base=1e4, scale=0.21, cap=20.0, v_mix=True, ff=72, limit=1.1):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot}, "scale": scale, "softcap": cap, "v_mix": v_mix},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=104, vocab=150, side=20, scale=3.0, eps=1e-5):
    return {"architecture": "Tepetar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "token_side": {"dim": side}, "layers": layers}


def uneven():
    """Every layer different: head counts, widths, windows, rotation, feed-forward; values first shared in layer 1."""
    return config([
        layer(heads=4, kv_heads=4, dim=48, vdim=32, window=17, rot=16, base=500.0, cap=5.0, v_mix=False, ff=None),
        layer(heads=6, kv_heads=2, dim=32, vdim=24, window=40, rot=32, scale=0.4),
        layer(heads=5, kv_heads=1, dim=80, vdim=56, window=1, rot=2, v_mix=False, ff=40, limit=0.4),
        layer(heads=2, kv_heads=2, dim=24, vdim=24, window=100, rot=12, base=7e5, cap=2.0, ff=200, limit=3.0),
        layer(heads=10, kv_heads=2, dim=16, vdim=24, window=33, rot=8, scale=1.0),
    ])


def shapes(cfg):
    w, v, s, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"], len(cfg["layers"])
    out = {"embed": (v, w), "side.embed": (v, n * s), "final.norm": (w,), "head": (v, w)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        hq, hk, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out |= {p + "norm1": (w,), p + "mix.q": (hq * d, w), p + "mix.q.b": (hq * d,), p + "mix.k": (hk * d, w), p + "mix.k.b": (hk * d,),
                p + "mix.v": (hk * e, w), p + "mix.v.b": (hk * e,), p + "mix.q.norm": (d,), p + "mix.k.norm": (d,), p + "mix.vmix": (),
                p + "mix.o": (w, hq * e), p + "mix.o.b": (w,), p + "side.gate": (s, w), p + "side.proj": (w, s), p + "side.norm": (w,)}
        if l["mlp"] is not None:
            f = l["mlp"]["ff"]
            out |= {p + "norm2": (w,), p + "mlp.gate": (f, w), p + "mlp.up": (f, w), p + "mlp.down": (w, f)}
    return out


def weights(cfg, seed=0):
    """bf16-representable float32 arrays under the source names."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith("vmix"):
            x = rng.uniform(0.2, 0.8)
        elif name.endswith((".norm", "norm1", "norm2")):
            plain = name.endswith(("q.norm", "k.norm", "side.norm"))
            x = (1 if plain else 0) + 0.3 * x
        elif name.endswith(".b"):
            x = 0.5 * x
        elif len(shape) == 2 and name not in ("embed", "side.embed"):
            x = x / np.sqrt(shape[1])
        out[name] = torch.as_tensor(np.asarray(x), dtype=torch.float32).bfloat16().float().numpy()
    return out


def write(path, cfg, tensors):
    """``config.json`` + ``model.safetensors`` (bfloat16) in ``path``."""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = torch.from_numpy(np.ascontiguousarray(t)).bfloat16().view(torch.uint8 if t.ndim else torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return path


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def spotlight(window, tail=3):
    """A one-layer model whose attention looks for token 1: its keys point along the query (a constant), those of every other
    token against it, and its value differs, so a logit shows at once whether token 1 is among the visible keys."""
    cfg = config([layer(heads=2, kv_heads=1, dim=16, vdim=16, window=window, rot=2, scale=1.0, cap=30.0, v_mix=True, ff=None)],
                 width=24, vocab=20, side=4)
    w = weights(cfg, 5)
    w["embed"][:, 0] = -1.0
    w["embed"][1, 0] = 1.0
    for n in ("l0.mix.q", "l0.mix.k"):
        w[n] = np.zeros_like(w[n])
    w["l0.mix.q.b"] = np.ones_like(w["l0.mix.q.b"])
    w["l0.mix.k.b"] = np.zeros_like(w["l0.mix.k.b"])
    w["l0.mix.k"][:, 0] = 1.0
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = np.ones(16, np.float32), np.ones(16, np.float32)
    w["l0.mix.v"][:, 0] = np.where(np.arange(16) % 2, 4.0, -4.0)
    return cfg, w

"""Small Kamedra checkpoints for the tests: configurations, seeded weights, and the directory form an engine loads."""

from __future__ import annotations

import numpy as np
import torch

from tepetar_cases import tokens, write  # noqa: F401  (any configuration with a vocabulary; any named tensors)

SCALING = {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 96}


def attention(heads=6, kv_heads=2, dim=20, vdim=24, window=40, keep=3, rot=16, base=1e4, scaling=None, scale=0.5, diff=0.35,
              ff=72, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep},
         "rot": {"base": base, "dims": rot, "scaling": scaling}, "scale": scale, "diff": diff}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def gla(heads=3, dim=24, vdim=40, tau=8.0, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=104, vocab=150, cap=12.0, eps=1e-5):
    return {"architecture": "Kamedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


def uneven():
    """Every layer different: kinds in no pattern, head counts, widths, windows, kept tokens, rotation, decay, feed-forward."""
    return config([
        gla(heads=3, dim=24, vdim=40, tau=4.0),
        attention(heads=4, kv_heads=2, dim=20, vdim=24, window=17, keep=5, rot=12, scaling=SCALING, diff=0.3),
        attention(heads=4, kv_heads=2, dim=20, vdim=24, window=50, keep=0, rot=12, scaling=SCALING, diff=0.8, scale=0.3, ff=None, kv_from=1),
        attention(heads=6, kv_heads=1, dim=48, vdim=80, window=1, keep=33, rot=48, base=500.0, scale=0.2, ff=40),
        gla(heads=2, dim=48, vdim=112, tau=1.0, ff=56),
        attention(heads=6, kv_heads=1, dim=48, vdim=80, window=100, keep=1, rot=48, base=500.0, scale=0.4, diff=0.6, ff=None, kv_from=3),
        attention(heads=10, kv_heads=1, dim=16, vdim=16, window=33, keep=16, rot=2, scale=0.7, ff=None),
    ])


def shapes(cfg, rank=lambda i: 8 + 12 * (i % 3)):
    w, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, w), "final.norm": (w,)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        out[p + "norm1"] = (w,)
        if l["type"] == "gla":
            h, d, e = m["heads"], m["dim"], m["vdim"]
            out |= {p + "mix.q": (h * d, w), p + "mix.k": (h * d, w), p + "mix.v": (h * e, w), p + "mix.g": (h * e, w), p + "mix.o": (w, h * e),
                    p + "mix.norm": (e,), p + "mix.a1": (rank(i), w), p + "mix.a2": (h * d, rank(i)), p + "mix.a2.b": (h * d,)}
        else:
            h, g, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out |= {p + "mix.q": (2 * h * d, w), p + "mix.o": (w, h * e), **{p + f"mix.{n}": (d,) for n in ("lq1", "lk1", "lq2", "lk2")}}
            if m.get("kv_from") is None:
                out |= {p + "mix.k": (2 * g * d, w), p + "mix.v": (g * e, w)}
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
        if name.endswith((".norm", "norm1", "norm2")):
            x = 1 + 0.3 * x
        elif name.endswith("a2.b"):
            x = 2.0 + 1.5 * x
        elif name.endswith(("lq1", "lk1", "lq2", "lk2")):
            x = x / np.sqrt(shape[0])
        elif name.endswith(("mix.k", "mix.q")):
            x = 1.2 * x / np.sqrt(shape[1])
        elif name == "embed":
            x = 0.3 * x  # small, so that the layers decide the logits (the table is also the output projection)
        elif len(shape) == 2:
            x = x / np.sqrt(shape[1])
        out[name] = bf16(x)
    for i, l in enumerate(cfg["layers"]):
        if l["type"] == "gla":  # keys lean towards queries: a first token's output is sign(q . k) v, which must not hang on rounding
            out[f"l{i}.mix.k"] = bf16(0.8 * out[f"l{i}.mix.q"] + 0.6 * out[f"l{i}.mix.k"])
    return out


def bf16(x):
    return torch.as_tensor(np.asarray(x), dtype=torch.float32).bfloat16().float().numpy()


def spotlight(window, keep, shared=False):
    """Attention whose first map looks for token 1 and whose second map is uniform: token 1's value differs, so a logit shows at
    once whether it is among the visible keys.  ``shared``: the looking is done by a second layer that reads the first one's pages
    (the first sees one token)."""
    looks = attention(heads=2, kv_heads=1, dim=16, vdim=16, window=window, keep=keep, rot=2, scale=1.0, diff=0.25, ff=None)
    layers = [looks]
    if shared:
        layers = [attention(heads=2, kv_heads=1, dim=16, vdim=16, window=1, keep=0, rot=2, scale=1.0, diff=0.5, ff=None), looks]
        looks["mixer"]["kv_from"] = 0
    cfg = config(layers, width=24, vocab=20)
    w = weights(cfg, 5)
    w["embed"] = bf16(0.2 * w["embed"])
    w["embed"][:, 0], w["embed"][:, 1] = -1.0, 1.0  # channel 0 marks token 1, channel 1 is constant
    w["embed"][1, 0] = 1.0
    for n in w:
        if n.endswith("norm1"):
            w[n] = np.ones_like(w[n])
        if n.endswith(("mix.q", "mix.k")):
            w[n] = np.zeros_like(w[n])
        if n.endswith("mix.o") and shared and n.startswith("l0"):
            w[n] = np.zeros_like(w[n])
    last = len(layers) - 1
    rows = np.arange(2, 16)  # channels that are not rotated
    for h in range(2):
        w[f"l{last}.mix.q"][h * 32 + rows, 1] = 1.0
    w["l0.mix.k"][rows, 0] = 1.0
    w["l0.mix.v"][:, 0] = np.where(np.arange(16) % 2, 2.0, -1.0)
    return cfg, w


def memory(dim=32, vdim=48):
    """One linear layer that forgets slowly (its decays stay near one), so that the first tokens reach far."""
    cfg = config([gla(heads=2, dim=dim, vdim=vdim, tau=16.0)], width=40, vocab=30)
    w = weights(cfg, 7)
    w["l0.mix.a2.b"] = bf16(np.full_like(w["l0.mix.a2.b"], 4.0))
    return cfg, w

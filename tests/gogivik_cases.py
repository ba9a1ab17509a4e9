"""Small Gogivik checkpoints for the tests: configurations, seeded weights, and models that make one mechanism stand out."""

from __future__ import annotations

import numpy as np

from bufolorn_cases import bf16
from tepetar_cases import tokens, write  # noqa: F401  (any configuration with a vocabulary; any named tensors)


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def latent(heads=3, dim=20, rot=12, vdim=28, q_rank=36, rank=40, window=24, scale=0.35, base=1e4, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": scale, "mask": {"size": window},
        "rot": {"base": base, "dims": rot}}}


def chunked(heads=6, kv_heads=2, dim=24, vdim=28, size=21, rot=16, base=300.0, factor=2.5, scale=0.4, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
        "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}}}


def mamba(heads=4, groups=2, state=24, vdim=20, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}}


def config(layers, width=104, vocab=150, taps=4, logit_scale=0.7, eps=1e-4):
    return {"architecture": "Gogivik", "vocab": vocab, "width": width, "canon": {"taps": taps}, "logit_scale": logit_scale, "norm": {"eps": eps},
            "layers": layers}


def uneven():
    """Every layer different: kinds in no pattern, head counts, widths, windows, chunks, ranks, rotation, taps, groups, feed-forwards."""
    return config([
        chunked(mlp=dense(40)),
        mamba(heads=6, groups=3, state=20, vdim=12, conv=2, norm_groups=4, mlp=dense()),
        latent(mlp=dense(56)),
        latent(heads=18, dim=8, rot=20, vdim=12, q_rank=70, rank=24, window=17, base=500.0, scale=0.2),
        mamba(heads=5, groups=1, state=48, vdim=40, conv=5, norm_groups=1),
        chunked(heads=4, kv_heads=1, dim=36, vdim=22, size=50, rot=36, base=7e3, factor=1.0, scale=0.2),
        chunked(heads=3, kv_heads=3, dim=20, vdim=48, size=7, rot=4, factor=6.0, mlp=dense(24)),
        mamba(heads=2, groups=2, state=16, vdim=72, conv=1, norm_groups=8, mlp=dense(32)),
        latent(heads=2, dim=24, rot=2, vdim=40, q_rank=16, rank=72, window=1, mlp=dense(24)),
    ])


def shapes(cfg):
    w, v, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    out = {"embed": (v, w), "final.norm": (w,), "head": (v, w)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        out |= {f"l{i}.norm1": (w,), f"l{i}.canon1": (w, taps)}
        if l["type"] == "latent_attention":
            h, d, r, e, a, c = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            out |= {p + "dq": (a, w), p + "dq.norm": (a,), p + "uq": (h * (d + r), a), p + "dkv": (c + r, w), p + "dkv.norm": (c,), p + "uk": (h * d, c),
                    p + "uv": (h * e, c), p + "sink": (h,), p + "o": (w, h * e)}
        elif l["type"] == "attention":
            h, g, d, e = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            out |= {p + "q": (h * d, w), p + "k": (g * d, w), p + "v": (g * e, w), p + "q.norm": (d,), p + "k.norm": (d,), p + "o": (w, h * e)}
        else:
            h, g, n, e = (m[k] for k in ("heads", "groups", "state", "vdim"))
            mixed = h * e + 2 * g * n
            out |= {p + "in": (h * e + mixed + h, w), p + "conv": (mixed, m["conv"]), p + "conv.b": (mixed,), p + "dt_bias": (h,), p + "A_log": (h,),
                    p + "D": (h,), p + "norm": (h * e,), p + "o": (w, h * e)}
        if l["mlp"] is not None:
            f = l["mlp"]["ff"]
            out |= {f"l{i}.norm2": (w,), f"l{i}.canon2": (w, taps), f"l{i}.mlp.up": (f, w), f"l{i}.mlp.down": (w, f)}
    return out


def weights(cfg, seed=0):
    """bf16-representable float32 arrays under the source names."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        x, last = rng.standard_normal(shape), name.split(".")[-1]
        if name == "final.norm" or last in ("norm1", "norm2"):
            x = 0.3 * x
        elif last == "norm":
            x = 1 + 0.3 * x
        elif last == "embed":
            x = 1.5 * x
        elif last in ("b", "A_log"):
            x = 0.4 * x
        elif last == "dt_bias":
            x = -1 + x
        elif last == "D":
            x = 1.2 + 0.3 * x
        elif last == "sink":
            x = 0.5 + x
        elif last in ("canon1", "canon2"):
            x = 0.3 * x
        elif last == "conv":
            x = 0.6 * x
        elif len(shape) == 2:
            x = x / np.sqrt(shape[1])
        out[name] = bf16(x)
    return out


def _marked(layer, taps=3):
    """Token 1 is marked in channel 0, channel 1 is constant; nothing but the layer's mixer changes the stream, and nothing mixes tokens
    in front of it."""
    cfg = config([layer], width=24, vocab=20, taps=taps, logit_scale=1.0)
    w = weights(cfg, 5)
    w["embed"] = bf16(0.1 * w["embed"])
    w["embed"][:, 0], w["embed"][:, 1] = -1.0, 1.0
    w["embed"][1, 0] = 1.0
    w["l0.norm1"], w["l0.canon1"] = np.zeros_like(w["l0.norm1"]), np.zeros_like(w["l0.canon1"])
    return cfg, w


def window_spotlight(window):
    """Latent attention that looks for token 1, whose value differs: a logit shows at once whether it is in the window."""
    cfg, w = _marked(latent(heads=2, dim=16, rot=2, vdim=16, q_rank=16, rank=16, window=window, scale=0.1))
    p = "l0.mix."
    for n in ("dq", "uq", "dkv", "uk", "uv"):
        w[p + n] = np.zeros_like(w[p + n])
    w[p + "dq"][:, 1], w[p + "dq.norm"], w[p + "dkv.norm"] = 1.0, np.ones(16, np.float32), np.ones(16, np.float32)
    for h in range(2):
        w[p + "uq"][h * 18 : h * 18 + 16, 0] = 1.0
    w[p + "dkv"][0, 0] = w[p + "dkv"][1, 1] = 1.0
    w[p + "uk"][:, 0] = 1.0
    w[p + "uv"][:, 0] = np.where(np.arange(32) % 2, 1.0, -0.5)
    return cfg, w


def chunk_spotlight(size):
    """Attention in chunks that looks for token 1: queries lean to a constant, its key along them and the other keys against them."""
    cfg, w = _marked(chunked(heads=2, kv_heads=1, dim=16, vdim=16, size=size, rot=2, scale=0.3))
    p = "l0.mix."
    for n in ("q", "k", "v"):
        w[p + n] = np.zeros_like(w[p + n])
    w[p + "q"][:, 1] = w[p + "k"][:, 0] = 1.0
    w[p + "q.norm"] = w[p + "k.norm"] = np.ones(16, np.float32)
    w[p + "v"][:, 0] = np.where(np.arange(16) % 2, 2.0, -1.0)
    return cfg, w


def memory():
    """A recurrence that forgets slowly, so that the first tokens reach far."""
    cfg = config([mamba(heads=2, groups=1, state=32, vdim=48, conv=3)], width=40, vocab=30)
    w = weights(cfg, 7)
    w["l0.mix.A_log"] = np.full_like(w["l0.mix.A_log"], -7.0)
    return cfg, w

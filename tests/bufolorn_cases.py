"""Small Bufolorn checkpoints for the tests: configurations, seeded weights, and models that make one mechanism stand out."""

from __future__ import annotations

import numpy as np
import torch

from tepetar_cases import tokens, write  # noqa: F401  (any configuration with a vocabulary; any named tensors)

SCALING = {"factor": 4.0, "original": 40, "fast": 4.0, "slow": 0.7}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, top=3, ff=40, shared=56, scale=1.6):
    out = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}
    return out | ({"shared": {"ff": shared}} if shared else {})


def latent(heads=3, dim=20, rot=12, vdim=28, rank=40, window=24, scale=0.35, base=1e4, scaling=SCALING, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": window},
         "rot": {"base": base, "dims": rot, "scaling": scaling}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel(heads=6, kv_heads=2, dim=20, vdim=28, bias_max=70, coef=0.4, every=16, scale=0.3, cap=9.0, rheads=3, rdim=24, scales=(0.9, 1.3), mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "scale": scale, "softcap": cap,
                 "q_temp": {"coef": coef, "every": every}},
        "right": {"heads": rheads, "dim": rdim}, "left_scale": scales[0], "right_scale": scales[1]}}


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=3, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(layers, width=104, vocab=150, embed=3.0, mult=0.6, eps=1e-4):
    return {"architecture": "Bufolorn", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "residual_mult": mult, "norm": {"eps": eps},
            "layers": layers}


def uneven():
    """Every layer different: kinds in no pattern, head counts, widths, windows, ranks, rotation, taps, feed-forwards."""
    return config([
        delta(heads=3, kv_heads=3, dim=20, vdim=28, conv=2, mlp=dense(40)),
        latent(mlp=moe()),
        parallel(),
        latent(heads=5, dim=48, vdim=16, window=50, kv_from=1, scale=0.2),
        delta(heads=4, kv_heads=2, dim=40, vdim=72, conv=5, mlp=moe(experts=5, top=1, shared=0, scale=0.8)),
        latent(heads=18, dim=8, rot=20, vdim=12, rank=24, window=17, scaling=None, base=300.0, mlp=dense(56)),
        parallel(heads=4, kv_heads=1, dim=36, vdim=20, bias_max=33, coef=0.2, every=5, cap=None, rheads=2, rdim=52, scales=(1.4, 0.7), mlp=moe(shared=24)),
        latent(heads=2, dim=24, vdim=40, window=1, kv_from=1, mlp=dense(24)),
    ])


def buckets(i):
    return 8 + 6 * (i % 3)


def shapes(cfg, rank=lambda i: 8 + 12 * (i % 3)):
    w, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, w), "final.norm": (w,), "final.norm.b": (w,), "head": (v, w)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        out |= {f"l{i}.norm1": (w,), f"l{i}.norm1.b": (w,)}
        if l["type"] == "latent_attention":
            h, d, r, e, c = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            out |= {p + "q": (h * (d + r), w), p + "uk": (h * d, c), p + "uv": (h * e, c), p + "o": (w, h * e)}
            if m.get("kv_from") is None:
                out |= {p + "dkv": (c + r, w), p + "dkv.norm": (c,)}
        elif l["type"] == "parallel":
            a, t = m["left"], m["right"]
            q = p + "left."
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out |= {q + n: (rows, w), q + n + ".b": (rows,)}
            out |= {q + "rel": (buckets(i), a["heads"]), q + "sink": (a["heads"],), q + "o": (w, a["heads"] * a["vdim"]), q + "o.b": (w,)}
            q, n = p + "right.", t["heads"] * t["dim"]
            out |= {q + "mu." + s: (w,) for s in "rkvgw"} | {q + s: (n, w) for s in "rkvg"}
            out |= {q + "w1": (rank(i), w), q + "w2": (n, rank(i)), q + "w0": (n,), q + "u": (t["heads"], t["dim"]), q + "norm": (n,), q + "o": (w, n)}
        else:
            h, g, d, e = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            for n, rows in (("q", g * d), ("k", g * d), ("v", h * e)):
                out |= {p + n: (rows, w), p + n + ".conv": (rows, m["conv"])}
            out |= {p + "b": (h, w), p + "A_log": (h,), p + "norm": (e,), p + "a1": (rank(i), w), p + "a2": (h * d, rank(i)), p + "dt_bias": (h * d,),
                    p + "g1": (rank(i + 1), w), p + "g2": (h * e, rank(i + 1)), p + "o": (w, h * e)}
        mlp, p = l["mlp"], f"l{i}.mlp."
        unit = lambda q, f: {q + "gate": (f, w), q + "up": (f, w), q + "down": (w, f)}
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out |= unit(p, mlp["ff"])
        else:
            for e in range(mlp["router"]["experts"]):
                out |= unit(f"{p}e{e}.", mlp["expert"]["ff"])
            out |= {p + "router": (mlp["router"]["experts"], w), p + "correction": (mlp["router"]["experts"],)}
            if mlp.get("shared"):
                out |= unit(p + "shared.", mlp["shared"]["ff"])
    return out


def weights(cfg, seed=0):
    """bf16-representable float32 arrays under the source names."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        x, last = rng.standard_normal(shape), name.split(".")[-1]
        if last in ("norm", "norm1"):
            x = 1 + 0.3 * x
        elif last == "b" and len(shape) == 1:
            x = 0.2 * x
        elif ".mu." in name:
            x = 1 / (1 + np.exp(-x))
        elif last == "w0":
            x = -2 + x
        elif last == "dt_bias":
            x = -1.5 + x
        elif last == "A_log":
            x = 0.5 * x
        elif last == "u":
            x = 0.3 + 0.4 * np.abs(x)
        elif last == "rel":
            x = 1.5 * x
        elif last == "sink":
            x = 0.5 + x
        elif last == "conv":
            x = 0.6 * x
        elif last == "correction":
            x = 0.2 * x
        elif last == "down":
            x = 0.7 * x / np.sqrt(shape[1])
        elif len(shape) == 2:
            x = x / np.sqrt(shape[1])
        out[name] = bf16(x)
    for i, l in enumerate(cfg["layers"]):  # keys lean towards queries: a first token's output is the sign of their product times v
        p = f"l{i}.mix."
        if l["type"] == "channel_delta":
            out[p + "k"] = bf16(0.8 * out[p + "q"] + 0.6 * out[p + "k"])
            out[p + "k.conv"] = bf16(0.8 * out[p + "q.conv"] + 0.6 * out[p + "k.conv"])
        elif l["type"] == "parallel":
            out[p + "right.k"] = bf16(0.8 * out[p + "right.r"] + 0.6 * out[p + "right.k"])
    return out


def bf16(x):
    return torch.as_tensor(np.asarray(x), dtype=torch.float32).bfloat16().float().numpy()


def _marked(layers):
    """Token 1 is marked in channel 0, channel 1 is constant; nothing but the last layer's mixer changes the stream."""
    cfg = config(layers, width=24, vocab=20, embed=1.0, mult=1.0)
    w = weights(cfg, 5)
    w["embed"] = bf16(0.2 * w["embed"])
    w["embed"][:, 0], w["embed"][:, 1] = -1.0, 1.0
    w["embed"][1, 0] = 1.0
    for n in w:
        if n.endswith("norm1"):
            w[n] = np.ones_like(w[n])
        if n.endswith("norm1.b"):
            w[n] = np.zeros_like(w[n])
    return cfg, w


def spotlight(window, shared=False):
    """Latent attention that looks for token 1, whose value differs: a logit shows at once whether it is in the window.  ``shared``: the
    looking is done by a second layer that reads the first one's latents (the first sees one token and adds nothing)."""
    looks = latent(heads=2, dim=16, rot=2, vdim=16, rank=16, window=window, scale=0.3, scaling=None)
    layers = [looks]
    if shared:
        layers = [latent(heads=2, dim=16, rot=2, vdim=16, rank=16, window=1, scale=0.3, scaling=None), looks]
        looks["mixer"]["kv_from"] = 0
    cfg, w = _marked(layers)
    for n in w:
        if n.endswith(("mix.q", "mix.dkv")):
            w[n] = np.zeros_like(w[n])
        if n == "l0.mix.o" and shared:
            w[n] = np.zeros_like(w[n])
    p = f"l{len(layers) - 1}.mix."
    for h in range(2):
        w[p + "q"][h * 18 : h * 18 + 16, 1] = 1.0
    w["l0.mix.dkv"][0, 0] = w["l0.mix.dkv"][1, 1] = 1.0
    w["l0.mix.dkv.norm"] = np.ones_like(w["l0.mix.dkv.norm"])
    w[p + "uk"], w[p + "uv"] = np.zeros_like(w[p + "uk"]), np.zeros_like(w[p + "uv"])
    w[p + "uk"][:, 0] = 0.5
    w[p + "uv"][:, 0] = np.where(np.arange(32) % 2, 1.0, -0.5)
    return cfg, w


def by_distance(bias_max, rows):
    """A parallel layer whose attention scores are the distance bias alone (queries are zero), with neighbouring buckets far apart, and
    whose time mixing adds nothing."""
    cfg, w = _marked([parallel(heads=2, kv_heads=1, dim=16, vdim=16, bias_max=bias_max, rheads=1, rdim=16, scales=(1.0, 1.0))])
    p = "l0.mix.left."
    for n in ("q", "q.b", "v.b", "o.b", "v"):
        w[p + n] = np.zeros_like(w[p + n])
    w[p + "v"][:, 0] = np.where(np.arange(16) % 2, 2.0, -1.0)
    w[p + "rel"] = bf16(np.array([[(3.0 if b % 2 else -3.0) + 0.25 * b, 0.2 * b] for b in range(rows)]))
    w["l0.mix.right.o"] = np.zeros_like(w["l0.mix.right.o"])
    return cfg, w


def far_key():
    """A parallel layer whose attention looks for token 1 however far back it is."""
    cfg, w = _marked([parallel(heads=2, kv_heads=1, dim=16, vdim=16, bias_max=40, coef=0.3, every=20, scale=0.5, cap=30.0, rheads=1, rdim=16)])
    p = "l0.mix.left."
    for n in ("q", "k", "q.b", "k.b", "v.b", "v"):
        w[p + n] = np.zeros_like(w[p + n])
    w[p + "q"][:, 1] = w[p + "k"][:, 0] = 1.0
    w[p + "v"][:, 0] = np.where(np.arange(16) % 2, 2.0, -1.0)
    w[p + "rel"] = bf16(0.3 * w[p + "rel"])
    w["l0.mix.right.o"] = np.zeros_like(w["l0.mix.right.o"])
    return cfg, w


def memory(kind):
    """One recurrent layer that forgets slowly, so that the first tokens reach far."""
    if kind == "delta":
        cfg = config([delta(heads=2, kv_heads=1, dim=32, vdim=48, conv=4)], width=40, vocab=30)
        w = weights(cfg, 7)
        w["l0.mix.dt_bias"] = np.full_like(w["l0.mix.dt_bias"], -9.0)
    else:
        cfg = config([parallel(rheads=2, rdim=32, scales=(0.1, 1.5))], width=40, vocab=30)
        w = weights(cfg, 7)
        w["l0.mix.right.w0"] = np.full_like(w["l0.mix.right.w0"], -7.0)
        w["l0.mix.right.w2"] = bf16(0.1 * w["l0.mix.right.w2"])
    return cfg, w

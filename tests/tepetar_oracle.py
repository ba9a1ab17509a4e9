"""Plain, slow restatement of the Tepetar decoder: one function per mechanism, numpy only, one sequence at a time.

Nothing here is shared with the product path.  ``dt`` chooses the arithmetic (float64 by default, so that the rounding of
this file never matters).  A model is ``(config dict, {tensor name: array})`` in the source names of its checkpoint.
"""

from __future__ import annotations

import numpy as np


def rms(x, eps):
    """x divided by its root mean square (last axis)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_centered(x, w, eps):
    """RMS norm whose stored weight is an offset from one."""
    return rms(x, eps) * (1 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def linear(x, w, b=None):
    y = x @ w.T
    return y if b is None else y + b


def rotate(x, positions, base, dims):
    """``x [T, heads, dim]``: channel i < dims/2 turns together with channel i + dims/2 by positions * base^(-2i/dims)."""
    half = dims // 2
    f = np.float64(base) ** (-2 * np.arange(half, dtype=np.float64) / dims) if half else np.zeros(0)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f
    c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def softcap(s, cap):
    return cap * np.tanh(s / cap)


def visible(qpos, kpos, window):
    d = np.asarray(qpos)[:, None] - np.asarray(kpos)[None]
    return (d >= 0) & (d < window)


def attend(q, k, v, qpos, kpos, scale, cap, window):
    """``q [Tq, H, d]``, ``k [Tk, G, d]``, ``v [Tk, G, e]`` -> ``[Tq, H, e]``; query head h reads group h // (H / G)."""
    tq, heads, _ = q.shape
    per = heads // k.shape[1]
    see = visible(qpos, kpos, window)
    out = np.zeros((tq, heads, v.shape[2]), dtype=q.dtype)
    for h in range(heads):
        s = softcap((q[:, h] @ k[:, h // per].T) * scale, cap)
        s = np.where(see, s, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (p / p.sum(-1, keepdims=True)) @ v[:, h // per]
    return out


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def clipped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g / (1 + np.exp(-1.702 * g)) * (u + 1)


def feed_forward(x, w, pre, mlp):
    limit = mlp["limit"]
    return linear(clipped_glu(linear(x, w[pre + "mlp.gate"]), linear(x, w[pre + "mlp.up"]), limit), w[pre + "mlp.down"])


def token_side(x, tokens, w, pre, layer, dim, eps):
    """What a layer's own slice of the per-token table adds to the stream."""
    e = w["side.embed"][tokens, layer * dim : (layer + 1) * dim]
    y = linear(gelu_tanh(linear(x, w[pre + "side.gate"])) * e, w[pre + "side.proj"])
    return norm_plain(y, w[pre + "side.norm"], eps)


class Model:
    """A sequence-at-a-time decoder.  ``state`` carries the keys, values and the count of tokens between portions."""

    def __init__(self, config, weights, dt=np.float64):
        self.cfg, self.dt = config, dt
        self.w = {k: np.asarray(v).astype(dt) for k, v in weights.items()}
        mixed = [i for i, l in enumerate(config["layers"]) if l["mixer"].get("v_mix")]
        self.first_mixed = mixed[0] if mixed else -1

    def start(self):
        return {"n": 0, "k": [None] * len(self.cfg["layers"]), "v": [None] * len(self.cfg["layers"])}

    def mixer(self, x, i, pos, state, first):
        m, w, p, eps = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", self.cfg["norm"]["eps"]
        t = len(x)
        q = linear(x, w[p + "q"], w[p + "q.b"]).reshape(t, m["heads"], m["dim"])
        k = linear(x, w[p + "k"], w[p + "k.b"]).reshape(t, m["kv_heads"], m["dim"])
        v = linear(x, w[p + "v"], w[p + "v.b"]).reshape(t, m["kv_heads"], m["vdim"])
        q = rotate(norm_plain(q, w[p + "q.norm"], eps), pos, m["rot"]["base"], m["rot"]["dims"])
        k = rotate(norm_plain(k, w[p + "k.norm"], eps), pos, m["rot"]["base"], m["rot"]["dims"])
        if m.get("v_mix"):
            if i == self.first_mixed:
                first = v
            else:
                v = mix_values(v, first, w[p + "vmix"])
        k = k if state["k"][i] is None else np.concatenate([state["k"][i], k])
        v = v if state["v"][i] is None else np.concatenate([state["v"][i], v])
        state["k"][i], state["v"][i] = k, v
        o = attend(q, k, v, pos, np.arange(len(k)), m["scale"], m["softcap"], m["mask"]["size"])
        return linear(o.reshape(t, -1), w[p + "o"], w[p + "o.b"]), first

    def run(self, tokens, state=None, trace=None):
        """Logits ``[T, vocab]`` of the next ``tokens`` of a sequence.  ``trace``: a list that gets the stream per layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        state = self.start() if state is None else state
        tokens = np.asarray(tokens)
        pos = state["n"] + np.arange(len(tokens))
        x = w["embed"][tokens] * self.dt(cfg["embedding"]["scale"])
        first = None
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            y, first = self.mixer(x, i, pos, state, first)
            x = x + norm_centered(y, w[p + "norm1"], eps)
            if layer["mlp"] is not None:
                x = x + norm_centered(feed_forward(x, w, p, layer["mlp"]), w[p + "norm2"], eps)
            x = x + token_side(x, tokens, w, p, i, cfg["token_side"]["dim"], eps)
            if trace is not None:
                trace.append(x)
        state["n"] += len(tokens)
        return linear(norm_centered(x, w["final.norm"], eps), w["head"])

    def generate(self, prompt, count):
        state, out = self.start(), []
        logits = self.run(prompt, state)
        for _ in range(count):
            out.append(int(logits[-1].argmax()))
            logits = self.run(out[-1:], state)
        return out

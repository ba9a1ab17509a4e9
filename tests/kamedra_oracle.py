"""Plain, slow restatement of the Kamedra decoder: one function per mechanism, numpy only, one sequence at a time.

Nothing here is shared with the product path.  ``dt`` chooses the arithmetic (float64 by default, so that the rounding of
this file never matters).  A model is ``(config dict, {tensor name: array})`` in the source names of its checkpoint.
"""

from __future__ import annotations

import numpy as np


def rms(x, eps):
    """x divided by its root mean square (last axis)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def softcap(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def frequencies(base, dims, scaling=None):
    """Rotation frequencies of the ``dims / 2`` pairs; ``scaling``: slow ones divided by a factor, with a linear blend between
    two wavelengths."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            turns = scaling["original"] * f / (2 * np.pi)  # rotations over the original context
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return np.array(out)


def rotate_pairs(x, positions, freq):
    """``x [T, heads, dim]``: channels 2i and 2i + 1 turn together by ``position * freq[i]``."""
    out = x.copy()
    for i, f in enumerate(freq):
        a = np.asarray(positions, dtype=np.float64) * f
        c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(qpos, kpos, window, keep):
    i, j = np.asarray(qpos)[:, None], np.asarray(kpos)[None]
    return (j <= i) & ((i - j < window) | (j < keep))


def attend(q, k, v, see, scale):
    """One head: ``q [Tq, d]``, ``k [Tk, d]``, ``v [Tk, e]``."""
    s = np.where(see, (q @ k.T) * scale, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def mixing_weight(lq1, lk1, lq2, lk2, diff):
    return np.exp((lq1 * lk1).sum()) - np.exp((lq2 * lk2).sum()) + diff


def difference(a1, a2, lam, diff, eps):
    """Second map subtracted from the first, per-head normalised."""
    return rms(a1 - lam * a2, eps) * (1 - diff)


def differential_attention(q, k, v, see, scale, lam, diff, eps):
    """``q [Tq, H, 2, d]``, ``k [Tk, G, 2, d]``, ``v [Tk, G, e]`` -> ``[Tq, H, e]``; head h reads group h // (H / G)."""
    heads = q.shape[1]
    per = heads // k.shape[1]
    out = np.zeros((q.shape[0], heads, v.shape[-1]), dtype=q.dtype)
    for h in range(heads):
        a1, a2 = (attend(q[:, h, m], k[:, h // per, m], v[:, h // per], see, scale) for m in (0, 1))
        out[:, h] = difference(a1, a2, lam, diff, eps)
    return out


def key_decay(h, a1, a2, bias, tau):
    return sigmoid((h @ a1.T) @ a2.T + bias) ** (1.0 / tau)


def gated_linear_attention(q, k, v, alpha, state):
    """``q, k, alpha [T, heads, d]``, ``v [T, heads, e]``; ``state [heads, d, e]`` is advanced in place."""
    out = np.zeros(v.shape, dtype=v.dtype)
    for t in range(len(q)):
        for n in range(q.shape[1]):
            state[n] = alpha[t, n][:, None] * state[n] + np.outer(k[t, n], v[t, n])
            out[t, n] = state[n].T @ q[t, n]
    return out


def feed_forward(h, w, pre):
    return (gelu_tanh(h @ w[pre + "mlp.gate"].T) * (h @ w[pre + "mlp.up"].T)) @ w[pre + "mlp.down"].T


class Model:
    """A sequence-at-a-time decoder.  The state carries keys, values, recurrent states and the count of tokens."""

    def __init__(self, config, weights, dt=np.float64):
        self.cfg, self.dt = config, dt
        self.w = {k: np.asarray(v).astype(dt) for k, v in weights.items()}

    def start(self):
        return {"n": 0, "k": {}, "v": {}, "s": {}}

    def attention(self, h, i, pos, state):
        m, w, p, eps = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", self.cfg["norm"]["eps"]
        t, d, e, g = len(h), m["dim"], m["vdim"], m["kv_heads"]
        rot = m.get("rot") or {"base": 1.0, "dims": 0}
        freq = frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        q = rotate_pairs((h @ w[p + "q"].T).reshape(t, m["heads"] * 2, d), pos, freq).reshape(t, m["heads"], 2, d)
        src = m.get("kv_from")
        if src is None:
            k = rotate_pairs((h @ w[p + "k"].T).reshape(t, g * 2, d), pos, freq).reshape(t, g, 2, d)
            v = (h @ w[p + "v"].T).reshape(t, g, e)
            state["k"][i] = np.concatenate([state["k"][i], k]) if i in state["k"] else k
            state["v"][i] = np.concatenate([state["v"][i], v]) if i in state["v"] else v
            src = i
        k, v = state["k"][src], state["v"][src]
        see = visible(pos, np.arange(len(k)), m["mask"]["size"], m["mask"].get("keep_first", 0))
        lam = mixing_weight(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
        o = differential_attention(q, k, v, see, m["scale"], lam, m["diff"], eps)
        return o.reshape(t, -1) @ w[p + "o"].T

    def gla(self, h, i, state):
        m, w, p, eps = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", self.cfg["norm"]["eps"]
        t, n, d, e = len(h), m["heads"], m["dim"], m["vdim"]
        q = (h @ w[p + "q"].T).reshape(t, n, d) * self.dt(d) ** self.dt(-0.5)
        k, v = (h @ w[p + "k"].T).reshape(t, n, d), (h @ w[p + "v"].T).reshape(t, n, e)
        alpha = key_decay(h, w[p + "a1"], w[p + "a2"], w[p + "a2.b"], m["tau"]).reshape(t, n, d)
        if i not in state["s"]:
            state["s"][i] = np.zeros((n, d, e), dtype=self.dt)
        o = norm(gated_linear_attention(q, k, v, alpha, state["s"][i]), w[p + "norm"], eps)
        z = h @ w[p + "g"].T
        return (o.reshape(t, -1) * z * sigmoid(z)) @ w[p + "o"].T

    def run(self, tokens, state=None, trace=None):
        """Logits ``[T, vocab]`` of the next ``tokens`` of a sequence.  ``trace``: a list that gets the stream per layer."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        state = self.start() if state is None else state
        tokens = np.asarray(tokens)
        pos = state["n"] + np.arange(len(tokens))
        x = w["embed"][tokens]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = norm(x, w[p + "norm1"], eps)
            x = x + (self.gla(h, i, state) if layer["type"] == "gla" else self.attention(h, i, pos, state))
            if layer["mlp"] is not None:
                x = x + feed_forward(norm(x, w[p + "norm2"], eps), w, p)
            if trace is not None:
                trace.append(x)
        state["n"] += len(tokens)
        return softcap(norm(x, w["final.norm"], eps) @ w["embed"].T, cfg.get("logit_softcap"))

    def generate(self, prompt, count):
        state, out = self.start(), []
        logits = self.run(prompt, state)
        for _ in range(count):
            out.append(int(logits[-1].argmax()))
            logits = self.run(out[-1:], state)
        return out

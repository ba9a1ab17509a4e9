"""Plain, slow restatement of the Bufolorn decoder: one function per mechanism, numpy only, one sequence at a time.

Nothing here is shared with the product path.  ``dt`` chooses the arithmetic (float64 by default, so that the rounding of
this file never matters).  A model is ``(config dict, {tensor name: array})`` in the source names of its checkpoint.
"""

from __future__ import annotations

import math

import numpy as np


# -- elementwise ----------------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0, z)


def rms(x, eps):
    """x divided by its root mean square (last axis)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdims=True)
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * w + b


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


# -- rotation -------------------------------------------------------------------------------------------------------
def frequencies(base, dims, scaling=None):
    """``(frequency of every pair, length of the rotated pair)``; ``scaling``: frequencies blend from kept to divided by a factor
    between the pairs that turn ``fast`` and ``slow`` times over the original context."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    place = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(place(scaling["fast"])), 0), min(math.ceil(place(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(scaling["factor"]) + 1


def rotate_pairs(x, positions, freq, length=1.0):
    """``x [T, heads, 2 * len(freq)]``: channels 2i and 2i + 1 turn together by ``position * freq[i]``."""
    out = x.copy()
    for i, f in enumerate(freq):
        a = np.asarray(positions, dtype=np.float64) * f
        c, s = (length * np.cos(a))[:, None].astype(x.dtype), (length * np.sin(a))[:, None].astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# -- attention ------------------------------------------------------------------------------------------------------
def visible(qpos, kpos, window=None):
    n = np.asarray(qpos)[:, None] - np.asarray(kpos)[None]
    return (n >= 0) & (n < window) if window else n >= 0


def temperature(positions, coef, every):
    return 1 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1) / every) + 1)


def bucket(n, rows, most):
    """Row of the distance table for a key ``n`` tokens back: one each up to half the rows, then logarithmic up to ``most``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(most / half) * (rows - half)))


def softcap(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def attend(scores, see, v, sink=None):
    """One head: ``scores [Tq, Tk]``, ``v [Tk, e]``; ``sink``: one more term of the denominator."""
    s = np.where(see, scores, -np.inf)
    top = s.max(-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    p = np.exp(s - top)
    total = p.sum(-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return (p / total) @ v


# -- recurrences ----------------------------------------------------------------------------------------------------
def short_conv(x, history, w):
    """``x [T, C]`` after the ``taps - 1`` inputs in ``history``; ``w [C, taps]``, last column for the current token.  Returns the
    result and the new history."""
    taps = w.shape[1]
    full = np.concatenate([history, x])
    y = sum(full[j : j + len(x)] * w[:, j] for j in range(taps))
    return y, full[len(full) - (taps - 1) :]


def delta_decay(h, a1, a2, dt_bias, a_log, heads):
    z = ((h @ a1.T) @ a2.T + dt_bias).reshape(len(h), heads, -1)
    return np.exp(-np.exp(a_log)[:, None] * softplus(z))


def delta_rule(q, k, v, beta, g, state):
    """``q, k, g [T, heads, d]``, ``v [T, heads, e]``, ``beta [T, heads]``; ``state [heads, d, e]`` is advanced in place."""
    out = np.zeros(v.shape, dtype=v.dtype)
    for t in range(len(q)):
        for n in range(q.shape[1]):
            s = g[t, n][:, None] * state[n]
            s = s + np.outer(k[t, n], beta[t, n] * (v[t, n] - s.T @ k[t, n]))
            state[n], out[t, n] = s, s.T @ q[t, n]
    return out


def shifted(h, last):
    """The previous token's row of every row; ``last``: what precedes the first."""
    return np.concatenate([last[None], h[:-1]])


def mixed(h, prev, mu):
    return h + (prev - h) * mu


def rwkv_decay(mix, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(mix @ w1.T) @ w2.T + w0))


def rwkv_rule(r, k, v, w, u, state):
    """``r, k, w [T, heads, d]``, ``v [T, heads, e]``, bonus ``u [heads, d]``; ``state [heads, d, e]`` is advanced in place."""
    out = np.zeros(v.shape, dtype=v.dtype)
    for t in range(len(r)):
        for n in range(r.shape[1]):
            kv = np.outer(k[t, n], v[t, n])
            out[t, n] = (state[n] + u[n][:, None] * kv).T @ r[t, n]
            state[n] = w[t, n][:, None] * state[n] + kv
    return out


# -- feed-forward ---------------------------------------------------------------------------------------------------
def gated_unit(h, gate, up, down, act):
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, correction, top, scale):
    """``(chosen experts [T, top], their weights)``."""
    s = sigmoid(h @ router.T)
    ids = np.argsort(-(s + correction), axis=-1, kind="stable")[:, :top]
    w = np.take_along_axis(s, ids, -1)
    return ids, w / (w.sum(-1, keepdims=True) + 1e-20) * scale


class Model:
    """A sequence-at-a-time decoder.  The state carries latents, keys, values, recurrent states and the count of tokens."""

    def __init__(self, config, weights, dt=np.float64):
        self.cfg, self.dt, self.eps = config, dt, config["norm"]["eps"]
        self.w = {k: np.asarray(v).astype(dt) for k, v in weights.items()}

    def start(self):
        return {"n": 0}

    @staticmethod
    def _append(state, key, rows):
        state[key] = np.concatenate([state[key], rows]) if key in state else rows
        return state[key]

    def _zeros(self, state, key, *shape):
        if key not in state:
            state[key] = np.zeros(shape, dtype=self.dt)
        return state[key]

    def latent_attention(self, h, i, pos, state):
        m, w, p, t = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", len(h)
        n, d, r, e, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        freq, length = frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
        q = (h @ w[p + "q"].T).reshape(t, n, d + r)
        q_rot = rotate_pairs(q[..., d:], pos, freq, length)
        src = m.get("kv_from")
        if src is None:
            row, src = h @ w[p + "dkv"].T, i
            self._append(state, ("c", i), rms(row[:, :rank], self.eps) * w[p + "dkv.norm"])
            self._append(state, ("r", i), rotate_pairs(row[:, None, rank:], pos, freq, length)[:, 0])
        c, k_rot = state["c", src], state["r", src]
        k, v = (c @ w[p + "uk"].T).reshape(-1, n, d), (c @ w[p + "uv"].T).reshape(-1, n, e)
        see = visible(pos, np.arange(len(c)), (m.get("mask") or {}).get("size"))
        o = [attend((q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"], see, v[:, a]) for a in range(n)]
        return np.concatenate(o, -1) @ w[p + "o"].T

    def biased_attention(self, h, m, p, i, pos, state):
        w, t = self.w, len(h)
        n, g, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        proj = lambda s: h @ w[p + s].T + w[p + s + ".b"]
        q = rms(proj("q").reshape(t, n, d), self.eps)
        if m.get("q_temp"):
            q = q * temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None].astype(self.dt)
        k = self._append(state, ("k", i), rms(proj("k").reshape(t, g, d), self.eps))
        v = self._append(state, ("v", i), proj("v").reshape(t, g, e))
        rel, dist = w[p + "rel"], pos[:, None] - np.arange(len(k))[None]
        rows = np.array([bucket(x, len(rel), m["bias_max"]) for x in range(len(k))])[np.maximum(dist, 0)]
        see, o = dist >= 0, []
        for a in range(n):
            s = softcap((q[:, a] @ k[:, a // (n // g)].T) * m["scale"], m.get("softcap")) + rel[rows, a]
            o.append(attend(s, see, v[:, a // (n // g)], w[p + "sink"][a]))
        return np.concatenate(o, -1) @ w[p + "o"].T + w[p + "o.b"]

    def time_mixing(self, h, m, p, i, state):
        w, t, n, d = self.w, len(h), m["heads"], m["dim"]
        prev = shifted(h, self._zeros(state, ("h", i), h.shape[1]))
        state["h", i] = h[-1]
        mix = {s: mixed(h, prev, w[p + "mu." + s]) for s in "rkvgw"}
        r, k, v = ((mix[s] @ w[p + s].T).reshape(t, n, d) for s in "rkv")
        decay = rwkv_decay(mix["w"], w[p + "w1"], w[p + "w2"], w[p + "w0"]).reshape(t, n, d)
        o = rwkv_rule(r, k, v, decay, w[p + "u"], self._zeros(state, ("s", i), n, d, d))
        return (rms(o, self.eps).reshape(t, -1) * w[p + "norm"] * silu(mix["g"] @ w[p + "g"].T)) @ w[p + "o"].T

    def parallel(self, h, i, pos, state):
        m, p = self.cfg["layers"][i]["mixer"], f"l{i}.mix."
        return (m["left_scale"] * self.biased_attention(h, m["left"], p + "left.", i, pos, state)
                + m["right_scale"] * self.time_mixing(h, m["right"], p + "right.", i, state))

    def channel_delta(self, h, i, state):
        m, w, p, t = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", len(h)
        n, g, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

        def conv(s):
            taps = w[p + s + ".conv"]
            y, state["c" + s, i] = short_conv(h @ w[p + s].T, self._zeros(state, ("c" + s, i), taps.shape[1] - 1, len(taps)), taps)
            return silu(y)
        q, k = (np.repeat(unit(conv(s).reshape(t, g, d)), n // g, 1) for s in "qk")
        v = conv("v").reshape(t, n, e)
        decay = delta_decay(h, w[p + "a1"], w[p + "a2"], w[p + "dt_bias"], w[p + "A_log"], n)
        o = delta_rule(q * d ** -0.5, k, v, sigmoid(h @ w[p + "b"].T), decay, self._zeros(state, ("s", i), n, d, e))
        gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
        return ((rms(o, self.eps) * w[p + "norm"]).reshape(t, -1) * gate) @ w[p + "o"].T

    def mixer(self, h, i, pos, state):
        kind = self.cfg["layers"][i]["type"]
        if kind == "latent_attention":
            return self.latent_attention(h, i, pos, state)
        return self.parallel(h, i, pos, state) if kind == "parallel" else self.channel_delta(h, i, state)

    def feed_forward(self, h, i):
        mlp, w, p = self.cfg["layers"][i]["mlp"], self.w, f"l{i}.mlp."
        if mlp["kind"] == "dense":
            return gated_unit(h, w[p + "gate"], w[p + "up"], w[p + "down"], lambda z: np.maximum(z, 0))
        unit_of = lambda rows, e: gated_unit(rows, w[p + e + ".gate"], w[p + e + ".up"], w[p + e + ".down"], silu)
        ids, weight = route(h, w[p + "router"], w[p + "correction"], mlp["router"]["top"], mlp["router"]["scale"])
        y = unit_of(h, "shared") if mlp.get("shared") else np.zeros_like(h)
        for e in range(mlp["router"]["experts"]):
            t, slot = np.nonzero(ids == e)
            y[t] += weight[t, slot][:, None] * unit_of(h[t], f"e{e}")
        return y

    def run(self, tokens, state=None, trace=None):
        """Logits ``[T, vocab]`` of the next ``tokens`` of a sequence.  ``trace``: a list that gets the stream per layer."""
        cfg, w = self.cfg, self.w
        state = self.start() if state is None else state
        tokens = np.asarray(tokens)
        pos = state["n"] + np.arange(len(tokens))
        x = w["embed"][tokens] * cfg["embedding"]["scale"]
        for i, layer in enumerate(cfg["layers"]):
            h = layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], self.eps)
            y = self.mixer(h, i, pos, state)
            if layer["mlp"] is not None:
                y = y + self.feed_forward(h, i)
            x = x + cfg["residual_mult"] * y
            if trace is not None:
                trace.append(x)
        state["n"] += len(tokens)
        return layer_norm(x, w["final.norm"], w["final.norm.b"], self.eps) @ w["head"].T

    def generate(self, prompt, count):
        state, out = self.start(), []
        logits = self.run(prompt, state)
        for _ in range(count):
            out.append(int(logits[-1].argmax()))
            logits = self.run(out[-1:], state)
        return out

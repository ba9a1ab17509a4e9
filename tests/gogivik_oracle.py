"""Plain, slow restatement of the Gogivik decoder: one function per mechanism, numpy only, one sequence at a time.

Nothing here is shared with the product path.  ``dt`` chooses the arithmetic (float64 by default, so that the rounding of
this file never matters).  A model is ``(config dict, {tensor name: array})`` in the source names of its checkpoint.
"""

from __future__ import annotations

import numpy as np


# -- elementwise ----------------------------------------------------------------------------------------------------
def silu(z):
    return z / (1 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0, z)


def rms(x, eps):
    """x divided by its root mean square (last axis)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_parts(x, parts, eps):
    """Every one of ``parts`` equal runs of channels divided by its own root mean square."""
    return rms(x.reshape(*x.shape[:-1], parts, -1), eps).reshape(x.shape)


def causal_conv(x, history, w):
    """``x [T, C]`` after the ``taps - 1`` inputs in ``history``; ``w [C, taps]``, last column for the current token.  Returns the
    result and the new history."""
    taps = w.shape[1]
    full = np.concatenate([history, x])
    y = sum(full[j : j + len(x)] * w[:, j] for j in range(taps))
    return y, full[len(full) - (taps - 1) :]


# -- rotation -------------------------------------------------------------------------------------------------------
def frequencies(base, dims, factor=1.0):
    return np.array([float(base) ** (-2.0 * i / dims) / factor for i in range(dims // 2)])


def turn(x, positions, freq, first, second):
    """``x [T, heads, d]``: channels ``first[i]`` and ``second[i]`` turn together by ``position * freq[i]``."""
    out = x.copy()
    for i, f in enumerate(freq):
        a = np.asarray(positions, dtype=np.float64) * f
        c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
        u, v = x[..., first[i]], x[..., second[i]]
        out[..., first[i]], out[..., second[i]] = u * c - v * s, v * c + u * s
    return out


def rotate_halves(x, positions, freq):
    """Channel i with channel i + half of the rotated ones."""
    n = len(freq)
    return turn(x, positions, freq, range(n), range(n, 2 * n))


def rotate_pairs(x, positions, freq):
    """Channel 2i with channel 2i + 1."""
    n = len(freq)
    return turn(x, positions, freq, range(0, 2 * n, 2), range(1, 2 * n, 2))


# -- attention ------------------------------------------------------------------------------------------------------
def in_window(qpos, kpos, size):
    n = np.asarray(qpos)[:, None] - np.asarray(kpos)[None]
    return (n >= 0) & (n < size)


def in_chunk(qpos, kpos, size):
    q, k = np.asarray(qpos)[:, None], np.asarray(kpos)[None]
    return (k <= q) & (q // size == k // size)


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


# -- recurrence -----------------------------------------------------------------------------------------------------
def state_space(x, b, c, dt, a_log, d, state):
    """``x [T, heads, e]``, ``b, c [T, heads, n]``, ``dt [T, heads]``; ``state [heads, n, e]`` is advanced in place."""
    out = np.zeros_like(x)
    for t in range(len(x)):
        keep = np.exp(-np.exp(a_log) * dt[t])
        state[:] = keep[:, None, None] * state + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out[t] = (state * c[t][:, :, None]).sum(1) + d[:, None] * x[t]
    return out


# -- feed-forward ---------------------------------------------------------------------------------------------------
def squared_unit(h, up, down):
    return np.maximum(h @ up.T, 0) ** 2 @ down.T


class Model:
    """A sequence-at-a-time decoder.  The state carries latents, keys, values, convolution inputs, recurrent states and the count of
    tokens."""

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

    def _conv(self, state, key, x, w):
        y, state[key] = causal_conv(x, self._zeros(state, key, w.shape[1] - 1, len(w)), w)
        return y

    def latent_attention(self, h, i, pos, state):
        m, w, p, t = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", len(h)
        n, d, r, e, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        freq = frequencies(m["rot"]["base"], m["rot"]["dims"])
        q = ((rms(h @ w[p + "dq"].T, self.eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(t, n, d + r)
        q_rot, row = rotate_pairs(q[..., d:], pos, freq), h @ w[p + "dkv"].T
        c = self._append(state, ("c", i), rms(row[:, :rank], self.eps) * w[p + "dkv.norm"])
        k_rot = self._append(state, ("r", i), rotate_pairs(row[:, None, rank:], pos, freq)[:, 0])
        k, v = (c @ w[p + "uk"].T).reshape(-1, n, d), (c @ w[p + "uv"].T).reshape(-1, n, e)
        see = in_window(pos, np.arange(len(c)), m["mask"]["size"])
        o = [attend((q[:, a, :d] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"], see, v[:, a], w[p + "sink"][a]) for a in range(n)]
        return np.concatenate(o, -1) @ w[p + "o"].T

    def attention(self, h, i, pos, state):
        m, w, p, t = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", len(h)
        n, g, d, e, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
        freq = frequencies(rot["base"], rot["dims"], (rot.get("scaling") or {"factor": 1.0})["factor"])
        vfreq = frequencies(rot["base"], e)
        q, k = (rotate_halves(rms((h @ w[p + s].T).reshape(t, -1, d), self.eps) * w[p + s + ".norm"], pos, freq) for s in "qk")
        k = self._append(state, ("k", i), k)
        v = self._append(state, ("v", i), rotate_halves(rms((h @ w[p + "v"].T).reshape(t, g, e), self.eps), pos, vfreq))
        see = in_chunk(pos, np.arange(len(k)), m["mask"]["size"])
        o = [attend((q[:, a] @ k[:, a // (n // g)].T) * m["scale"], see, v[:, a // (n // g)]) for a in range(n)]
        return rotate_halves(np.stack(o, 1), -pos, vfreq).reshape(t, -1) @ w[p + "o"].T

    def mamba2(self, h, i, state):
        m, w, p, t = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix.", len(h)
        n, e, s, g = m["heads"], m["vdim"], m["state"], m["groups"]
        z, xbc, dt = np.split(h @ w[p + "in"].T, [n * e, 2 * n * e + 2 * g * s], axis=1)
        xbc = silu(self._conv(state, ("conv", i), xbc, w[p + "conv"]) + w[p + "conv.b"])
        x, b, c = np.split(xbc, [n * e, n * e + g * s], axis=1)
        b, c = (np.repeat(u.reshape(t, g, s), n // g, 1) for u in (b, c))
        y = state_space(x.reshape(t, n, e), b, c, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"], self._zeros(state, ("s", i), n, s, e))
        return (rms_parts(y.reshape(t, -1) * silu(z), m["norm_groups"], self.eps) * w[p + "norm"]) @ w[p + "o"].T

    def mixer(self, h, i, pos, state):
        kind = self.cfg["layers"][i]["type"]
        if kind == "mamba2":
            return self.mamba2(h, i, state)
        return {"latent_attention": self.latent_attention, "attention": self.attention}[kind](h, i, pos, state)

    def sublayer_input(self, x, i, which, state):
        """What sublayer 1 or 2 of a layer reads: the normed stream plus its convolution over time."""
        h = rms(x, self.eps) * (1 + self.w[f"l{i}.norm{which}"])
        return h + self._conv(state, ("canon", which, i), h, self.w[f"l{i}.canon{which}"])

    def run(self, tokens, state=None, trace=None):
        """Logits ``[T, vocab]`` of the next ``tokens`` of a sequence.  ``trace``: a list that gets the stream per layer."""
        cfg, w = self.cfg, self.w
        state = self.start() if state is None else state
        tokens = np.asarray(tokens)
        pos = state["n"] + np.arange(len(tokens))
        x = w["embed"][tokens]
        for i, layer in enumerate(cfg["layers"]):
            x = x + self.mixer(self.sublayer_input(x, i, 1, state), i, pos, state)
            if layer["mlp"] is not None:
                x = x + squared_unit(self.sublayer_input(x, i, 2, state), w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"])
            if trace is not None:
                trace.append(x)
        state["n"] += len(tokens)
        return (rms(x, self.eps) * (1 + w["final.norm"])) @ w["head"].T * cfg["logit_scale"]

    def generate(self, prompt, count):
        state, out = self.start(), []
        logits = self.run(prompt, state)
        for _ in range(count):
            out.append(int(logits[-1].argmax()))
            logits = self.run(out[-1:], state)
        return out

"""Plain restatement of the Rumazen decoder in numpy, one function per mechanism, written for clarity and not for
speed (double precision by default).  Test infrastructure only: nothing of the product imports it.

A layer is parallel: x <- x + mixer(h) + ff(h) with h = norm(x).  The mixer is either softmax attention over a sliding
window plus pooled blocks that have left it, or a recurrence with a generalised delta rule.
Weights are a dict name -> array with the tensor names of a checkpoint; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    """x over its root mean square along the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_rms_norm(x, gain, eps):
    return rms(x, eps) * float(np.asarray(gain).reshape(()))


def rotate_interleaved(x, positions, dims, base, factor=1.0):
    """x [tokens, heads, dim]: coordinates (2i, 2i + 1), i < dims / 2, turned by position * base^(-2i/dims) / factor"""
    out = np.array(x, copy=True)
    for i in range(dims // 2):
        angle = np.asarray(positions, np.float64) * (base ** (-2.0 * i / dims) / factor)
        c, s = np.cos(angle)[:, None].astype(x.dtype), np.sin(angle)[:, None].astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(i, size, pool):
    """-> (first token seen by position i, number of pooled blocks it sees); the last token seen is i itself"""
    if not size:
        return 0, 0
    blocks = 0
    while pool and (blocks + 1) * pool - 1 <= i - size:
        blocks += 1
    return max(0, i - size + 1), blocks


def window_attention(q, k, v, scale, size=0, pool=0, softcap=0.0, first=0):
    """q [Tq, H, d] at positions first..first+Tq-1 over keys k [T, G, d] / values v [T, G, e] of positions 0..T-1
    -> [Tq, H, e]"""
    tq, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((tq, heads, v.shape[2]), q.dtype)
    nb = k.shape[0] // pool if pool else 0
    pk = [k[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]
    pv = [v[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]
    for t in range(tq):
        i = first + t
        lo, blocks = visible(i, size, pool)
        keys = np.stack(pk[:blocks] + [k[j] for j in range(lo, i + 1)])
        vals = np.stack(pv[:blocks] + [v[j] for j in range(lo, i + 1)])
        for h in range(heads):
            s = keys[:, h // group] @ q[t, h] * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ vals[:, h // group]
    return out


def delta_rule(r, k, v, w, a, state, unit_eps=1e-6):
    """r, k, v, w, a [T, H, d]; state [H, d(key), d(value)] -> (o [T, H, d], state after)"""
    state = np.array(state, copy=True)
    out = np.zeros_like(v)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            u = k[t, h] / np.sqrt(np.sum(k[t, h] ** 2) + unit_eps)
            old = state[h]
            seen = u @ old
            state[h] = w[t, h][:, None] * old - np.outer(a[t, h] * u, seen) + np.outer(k[t, h], v[t, h])
            out[t, h] = r[t, h] @ state[h]
    return out, state


def delta_decay(z):
    """decay from its pre-activation"""
    return np.exp(-np.exp(-0.5) * sigmoid(z))


class Model:
    def __init__(self, config, weights, dtype=np.float64):
        self.c = config
        self.w = {n: np.asarray(t, dtype) for n, t in weights.items()}
        self.dtype = dtype

    def attention(self, l, m, h):
        p, n = f"l{l}.mix.", h.shape[0]
        heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = (h @ self.w[p + "q"].T).reshape(n, heads, dim)
        k = (h @ self.w[p + "k"].T).reshape(n, kv, dim)
        v = (h @ self.w[p + "v"].T).reshape(n, kv, vdim)
        rot, mask = m.get("rot"), m.get("mask") or {}
        if rot:
            f = (rot.get("scaling") or {}).get("factor", 1.0)
            q = rotate_interleaved(q, np.arange(n), rot["dims"], rot["base"], f)
            k = rotate_interleaved(k, np.arange(n), rot["dims"], rot["base"], f)
        o = window_attention(q, k, v, m["scale"], mask.get("size", 0), mask.get("pool", 0), m.get("softcap") or 0.0)
        o = o * sigmoid(h @ self.w[p + "g"].T)[:, :, None]
        return o.reshape(n, heads * vdim) @ self.w[p + "o"].T

    def general_delta(self, l, m, h):
        p, n, shape = f"l{l}.mix.", h.shape[0], (h.shape[0], m["heads"], m["dim"])
        r, k, v = ((h @ self.w[p + x].T).reshape(shape) for x in "rkv")
        w = delta_decay(np.tanh(h @ self.w[p + "w1"].T) @ self.w[p + "w2"].T + self.w[p + "w0"]).reshape(shape)
        a = sigmoid(h @ self.w[p + "a"].T + self.w[p + "a.b"]).reshape(shape)
        o, _ = delta_rule(r, k, v, w, a, np.zeros((m["heads"], m["dim"], m["dim"]), self.dtype))
        o = rms(o, self.c["norm"]["eps"]).reshape(n, -1) * self.w[p + "norm"] * sigmoid(h @ self.w[p + "g"].T)
        return o @ self.w[p + "o"].T

    def feed_forward(self, l, h):
        p = f"l{l}.mlp."
        return (gelu_tanh(h @ self.w[p + "gate"].T) * (h @ self.w[p + "up"].T)) @ self.w[p + "down"].T

    def forward(self, ids, layers_out=None):
        """logits [tokens, vocab] of a whole sequence; layers_out (a list) receives the residual after every layer"""
        x = self.w["embed"][np.asarray(ids)] * self.c["embedding"]["scale"]
        for l, layer in enumerate(self.c["layers"]):
            h = scalar_rms_norm(x, self.w[f"l{l}.norm1"], self.c["norm"]["eps"])
            y = getattr(self, layer["type"])(l, layer["mixer"], h)
            if layer.get("mlp"):
                y = y + self.feed_forward(l, h)
            x = x + y
            if layers_out is not None:
                layers_out.append(x)
        return scalar_rms_norm(x, self.w["final.norm"], self.c["norm"]["eps"]) @ self.w["head"].T

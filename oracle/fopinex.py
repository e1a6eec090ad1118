"""Plain restatement of the Fopinex decoder in numpy, one function per mechanism, written for clarity and not for speed
(double precision by default).  Test infrastructure only: nothing of the product imports it.

A layer is parallel with a norm of its own for either branch, and both branches leave through an elementwise gate:
    x <- x + m (sigmoid(A1 h1 + b1) mixer(h1) + sigmoid(A2 h2 + b2) ff(h2))      h1, h2 = norm1(x), norm2(x)
The mixer is gated linear attention or attention with sigmoid weights that are mixed across heads, the feed-forward a
mixture of experts.  Weights are a dict name -> array with the tensor names of a checkpoint; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def gla_decay(z, tau):
    """decay of a key channel from its pre-activation"""
    return sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(q, k, v, decay, state):
    """q, k, decay [T, H, d], v [T, H, e], state [H, d, e] -> (o [T, H, e], state after)"""
    state, out = np.array(state, copy=True), np.zeros(v.shape, v.dtype)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            state[h] = decay[t, h][:, None] * state[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = q[t, h] @ state[h]
    return out, state


def chunk_start(i, size):
    """first position that position i sees"""
    return i - i % size if size else 0


def mixed_sigmoid_attention(q, k, v, scale, bias, talk, size=0, first=0):
    """q [Tq, H, d] at positions first..first+Tq-1 over keys k [T, G, d] / values v [T, G, e] of positions 0..T-1, weights
    sigmoid(scale q.k + bias) per head, then mixed by talk [H, H] -> [Tq, H, e]"""
    tq, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((tq, heads, v.shape[2]), q.dtype)
    for t in range(tq):
        lo, hi = chunk_start(first + t, size), first + t + 1
        w = np.stack([sigmoid(k[lo:hi, g // group] @ q[t, g] * scale + bias[g]) for g in range(heads)])
        w = talk @ w
        for h in range(heads):
            out[t, h] = w[h] @ v[lo:hi, h // group]
    return out


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(z, correction, top, groups=1, keep=1):
    """router logits z [n] of one token -> (chosen indexes, their weights)"""
    s = np.exp(z - z.max())
    s = s / s.sum()
    choice = s + correction
    n = len(z) // groups
    best = np.argsort(-choice.reshape(groups, n).max(1), kind="stable")[:keep]
    allowed = [e for e in range(len(z)) if e // n in best]
    chosen = sorted(allowed, key=lambda e: (-choice[e], e))[:top]
    return chosen, s[chosen]


class Model:
    def __init__(self, config, weights, dtype=np.float64):
        self.c = config
        self.w = {n: np.asarray(t, dtype) for n, t in weights.items()}
        self.dtype = dtype

    def gla(self, l, m, h):
        p, n, eps = f"l{l}.mix.", h.shape[0], self.c["norm"]["eps"]
        heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
        q = (h @ self.w[p + "q"].T).reshape(n, heads, dim) * dim ** -0.5
        k = (h @ self.w[p + "k"].T).reshape(n, heads, dim)
        v = (h @ self.w[p + "v"].T).reshape(n, heads, vdim)
        z = h @ self.w[p + "a1"].T @ self.w[p + "a2"].T + self.w[p + "a2.b"]
        o, _ = gated_linear_attention(q, k, v, gla_decay(z, m["tau"]).reshape(n, heads, dim), np.zeros((heads, dim, vdim), self.dtype))
        g = h @ self.w[p + "g"].T
        return (rms_norm(o, self.w[p + "norm"], eps).reshape(n, -1) * g * sigmoid(g)) @ self.w[p + "o"].T

    def attention(self, l, m, h, kv):
        p, n = f"l{l}.mix.", h.shape[0]
        heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = (h @ self.w[p + "q"].T).reshape(n, heads, dim)
        if m.get("kv_from") is None:
            kv[l] = ((h @ self.w[p + "k"].T).reshape(n, kv_heads, dim), (h @ self.w[p + "v"].T).reshape(n, kv_heads, vdim))
            k, v = kv[l]
        else:
            k, v = kv[m["kv_from"]]
        o = mixed_sigmoid_attention(q, k, v, m["scale"], self.w[p + "pb"], self.w[p + "talk"], (m.get("mask") or {}).get("size", 0))
        return o.reshape(n, heads * vdim) @ self.w[p + "o"].T

    def experts(self, l, f, h):
        p, r, limit = f"l{l}.mlp.", f["router"], f["expert"]["limit"]
        groups = r.get("groups") or {}
        z = h @ self.w[p + "router"].T
        out = np.zeros_like(h)
        for t in range(h.shape[0]):
            for e, s in zip(*route(z[t], self.w[p + "correction"], r["top"], groups.get("count", 1), groups.get("keep", 1))):
                y = h[t]
                if e < r["experts"]:
                    y = clamped_expert(h[t], *(self.w[f"{p}e{e}.{x}"] for x in ("gate", "up", "down")), limit)
                out[t] += s * y
        return out

    def forward(self, ids, layers_out=None):
        """logits [tokens, vocab] of a whole sequence; layers_out (a list) receives the residual after every layer"""
        eps, mult, kv = self.c["norm"]["eps"], self.c["residual_mult"], {}
        x = self.w["embed"][np.asarray(ids)]
        for l, layer in enumerate(self.c["layers"]):
            p = f"l{l}."
            h = rms_norm(x, self.w[p + "norm1"], eps)
            y = self.gla(l, layer["mixer"], h) if layer["type"] == "gla" else self.attention(l, layer["mixer"], h, kv)
            y = y * sigmoid(h @ self.w[p + "rg1"].T + self.w[p + "rg1.b"])
            if layer.get("mlp"):
                h = rms_norm(x, self.w[p + "norm2"], eps)
                y = y + self.experts(l, layer["mlp"], h) * sigmoid(h @ self.w[p + "rg2"].T + self.w[p + "rg2.b"])
            x = x + mult * y
            if layers_out is not None:
                layers_out.append(x)
        return rms_norm(x, self.w["final.norm"], eps) @ self.w["head"].T

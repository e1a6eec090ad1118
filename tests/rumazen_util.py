"""Small Rumazen configurations, random checkpoints, and ways to run them (test helper)."""
import json
import os
import struct

import numpy as np

from oracle import rumazen


def attention(heads, kv_heads, dim, vdim, rot=None, base=10000.0, factor=None, scale=None, softcap=None, size=None, pool=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5)
    if rot:
        m["rot"] = dict(dims=rot, base=base)
        if factor:
            m["rot"]["scaling"] = dict(factor=factor)
    if softcap:
        m["softcap"] = softcap
    if size:
        m["mask"] = dict(size=size)
        if pool:
            m["mask"]["pool"] = pool
    return m


def layer(kind, mixer, ff):
    return dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None)


def config(vocab, width, layers, eps=1e-5, scale=1.0):
    return dict(architecture="Rumazen", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


# sizes no power of two, every width different, a layer without feed-forward, two windows
ODD = config(331, 150, [
    layer("general_delta", dict(heads=3, dim=24), 87),
    layer("attention", attention(6, 2, 40, 28, rot=24, base=700.0, factor=2.5, scale=0.21, softcap=9.0, size=19, pool=5), 104),
    layer("general_delta", dict(heads=5, dim=12), 0),
    layer("attention", attention(4, 4, 36, 52, rot=36, base=5000.0, scale=0.15, softcap=40.0, size=33, pool=7), 0),
], eps=3e-5, scale=1.7)
# sizes the tensor-core kernels take
EVEN = config(512, 256, [
    layer("attention", attention(4, 2, 64, 64, rot=48, base=20000.0, factor=3.0, scale=0.11, softcap=20.0, size=150, pool=16), 192),
    layer("general_delta", dict(heads=3, dim=64), 256),
    layer("attention", attention(8, 1, 128, 128, rot=128, factor=1.5, scale=0.07, softcap=15.0, size=70, pool=4), 128),
    layer("general_delta", dict(heads=2, dim=128), 128),
])
# everything that can be one is one; no rotation, no cap, no pooling somewhere
ONES = config(64, 16, [
    layer("attention", attention(1, 1, 2, 1, rot=2, factor=1.0, scale=1.0, softcap=5.0, size=1, pool=1), 1),
    layer("general_delta", dict(heads=1, dim=1), 1),
    layer("attention", attention(2, 1, 8, 8, size=6), 8),
    layer("attention", attention(2, 2, 6, 4, rot=4), 24),
])


def bf16_round(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return (((u + 0x7fff + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def weights(cfg, seed=0, rank=9, sharp=1.0):
    """name -> float32 array that bf16 holds exactly; ``sharp`` scales q and k, for scores that stand out"""
    rng = np.random.default_rng(seed)
    w, width = {}, cfg["width"]

    def lin(name, rows, cols, gain=1.0):
        w[name] = bf16_round(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean, std):
        w[name] = bf16_round(mean + std * rng.standard_normal(n))

    lin("embed", cfg["vocab"], width, np.sqrt(width))
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        w[p + "norm1"] = bf16_round(rng.uniform(0.7, 1.4, ()))
        if l["type"] == "attention":
            lin(p + "mix.q", m["heads"] * m["dim"], width, 1.5 * sharp)
            lin(p + "mix.k", m["kv_heads"] * m["dim"], width, 1.5 * sharp)
            lin(p + "mix.v", m["kv_heads"] * m["vdim"], width)
            lin(p + "mix.g", m["heads"], width)
            lin(p + "mix.o", width, m["heads"] * m["vdim"])
        else:
            n = m["heads"] * m["dim"]
            for x in "rkvga":
                lin(p + "mix." + x, n, width)
            lin(p + "mix.w1", rank, width)
            lin(p + "mix.w2", n, rank)
            vec(p + "mix.w0", n, -1.0, 1.5)
            vec(p + "mix.a.b", n, 0.0, 1.0)
            vec(p + "mix.norm", n, 1.0, 0.2)
            lin(p + "mix.o", width, n)
        if l["mlp"]:
            lin(p + "mlp.gate", l["mlp"]["ff"], width)
            lin(p + "mlp.up", l["mlp"]["ff"], width)
            lin(p + "mlp.down", width, l["mlp"]["ff"])
    w["final.norm"] = bf16_round(rng.uniform(0.7, 1.4, ()))
    lin("head", cfg["vocab"], width)
    return w


def write_checkpoint(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, a in w.items():
        a = np.asarray(a, np.float32)
        raw = (np.ascontiguousarray(a).reshape(-1).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = dict(dtype="BF16", shape=list(a.shape), data_offsets=[at, at + len(raw)])
        at += len(raw)
        blobs.append(raw)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


def error(got, want):
    """per row: rms over the vocabulary of the difference without its mean, over the spread of the wanted logits"""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.std(want)


class Runner:
    """One model with slabs of its own, driven through prefill and decode."""

    def __init__(self, folder, dtype, slots=4, session_len=512, max_prefill_tokens=0, max_batch_size=8):
        import torch
        from lmdeploy_b200 import decoder
        self.model = decoder.Model.open(folder, dtype, max_batch_size, session_len, max_prefill_tokens)
        # garbage in the slabs: nothing may depend on what a slab held before
        self.slabs = [torch.full((self.model.slab_bytes,), 0x3f, dtype=torch.uint8, device="cuda") for _ in range(slots)]
        self.length = [0] * slots

    def reset(self, slot):
        self.length[slot] = 0

    def prefill(self, parts):
        """parts: slot -> tokens; logits of every token, per slot"""
        slots = list(parts)
        lg, _ = self.model.prefill([parts[s] for s in slots], [self.length[s] for s in slots], [self.slabs[s].data_ptr() for s in slots],
                                   [range(len(parts[s])) for s in slots])
        self.model.check_status()
        lg, out, at = lg.cpu().numpy(), {}, 0
        for s in slots:
            self.length[s] += len(parts[s])
            out[s] = lg[at:at + len(parts[s])]
            at += len(parts[s])
        return out

    def decode(self, tokens, use_graph=False):
        """tokens: slot -> one token; logits per slot"""
        slots = list(tokens)
        st = self.model.new_state([self.slabs[s].data_ptr() for s in slots], [self.length[s] for s in slots], 1, [[tokens[s] for s in slots]])
        self.model.decode(st, 1, use_graph)
        self.model.check_status()
        for s in slots:
            self.length[s] += 1
        lg = st.logits.cpu().numpy()
        return {s: lg[i] for i, s in enumerate(slots)}

    def close(self):
        self.model.close()


def first_token_margin(cfg, w, token):
    """At its first token a delta-rule head gives (r . k) v over its own root mean square, that is v with the SIGN of r . k:
    rounding decides where r and k are all but orthogonal.  -> the smallest |cos(r, k)| of any head for this first token."""
    seen = [1.0]
    m = rumazen.Model(cfg, w)
    mix = m.general_delta

    def watched(l, spec, h):
        r, k = ((h @ m.w[f"l{l}.mix.{x}"].T).reshape(spec["heads"], spec["dim"]) for x in "rk")
        seen.append(np.abs((r * k).sum(-1) / np.linalg.norm(r, axis=-1) / np.linalg.norm(k, axis=-1)).min())
        return mix(l, spec, h)

    m.general_delta = watched
    m.forward([token])
    return min(seen)


def prompts(cfg, w, lengths, seed=5):
    """random token ids whose first token is well conditioned (first_token_margin)"""
    rng, out = np.random.default_rng(seed), []
    for n in lengths:
        ids = list(map(int, rng.integers(0, cfg["vocab"], n)))
        while first_token_margin(cfg, w, ids[0]) < 0.02:
            ids[0] = int(rng.integers(0, cfg["vocab"]))
        out.append(ids)
    return out


def oracle_logits(cfg, w, ids):
    return rumazen.Model(cfg, w).forward(ids)

"""Small Fopinex configurations, random checkpoints, and the plain restatement of them (test helper)."""
import numpy as np

from oracle import fopinex
from tests.rumazen_util import Runner, bf16_round, error, write_checkpoint  # noqa: F401  (used by the tests)


def attention(heads, kv_heads, dim, vdim, size=None, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5)
    if size:
        m["mask"] = dict(size=size)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def gla(heads, dim, vdim, tau):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def moe(experts, top, ff, limit=2.0, identity=None, groups=None, keep=None):
    router = dict(experts=experts, top=top)
    if identity is not None:
        router["identity"] = identity
    if groups:
        router["groups"] = dict(count=groups, keep=keep)
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=router)


def layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def config(vocab, width, layers, eps=1e-5, mult=0.8):
    return dict(architecture="Fopinex", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult, layers=layers)


# sizes no power of two, every width different, layers without feed-forward, shared keys with another chunk than their
# owner's (longer and shorter) and not from the layer ahead, routers that choose
ODD = config(331, 150, [
    layer("attention", attention(6, 2, 20, 12, 19, 0.31), moe(5, 3, 27, 1.2, identity=3, groups=4, keep=2)),
    layer("gla", gla(3, 24, 20, 7.0), None),
    layer("attention", attention(6, 2, 20, 12, 47, 0.2, kv_from=0), moe(7, 2, 40, 0.9, identity=0)),
    layer("attention", attention(4, 4, 36, 52), None),
    layer("gla", gla(5, 12, 33, 16.0), moe(9, 4, 17, 3.0, identity=6, groups=3, keep=2)),
    layer("attention", attention(4, 4, 36, 52, 5, kv_from=3), moe(4, 1, 65, 1.5)),
], eps=3e-5, mult=0.6)
# sizes the tensor-core kernels take; routers that leave nothing to choose, so that 16 bits choose what fp32 does
EVEN = config(512, 256, [
    layer("attention", attention(8, 4, 64, 64, 150), moe(6, 8, 96, 1.7, identity=2)),
    layer("attention", attention(8, 4, 64, 64, 70, kv_from=0), moe(4, 4, 128)),
    layer("gla", gla(4, 64, 128, 12.0), moe(3, 4, 64, identity=1, groups=2, keep=2)),
    layer("attention", attention(16, 2, 128, 128, 200), None),
    layer("gla", gla(2, 128, 64, 5.0), moe(2, 2, 200, 1.0)),
    layer("attention", attention(20, 1, 72, 40), moe(1, 1, 64, 2.5)),
], mult=0.7)
# everything that can be one is one
ONES = config(64, 16, [
    layer("attention", attention(1, 1, 2, 1, 1, 1.0), moe(1, 1, 1, 1.0)),
    layer("gla", gla(1, 1, 1, 1.0), moe(1, 2, 1, 1.0, identity=1, groups=1, keep=1)),
    layer("attention", attention(2, 1, 8, 8, 6), None),
    layer("attention", attention(2, 1, 8, 8, kv_from=2), moe(2, 2, 8)),
    layer("attention", attention(1, 1, 8, 16), None),
], mult=1.0)


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
        vec(p + "norm1", width, 1.0, 0.2)
        if l["type"] == "attention":
            lin(p + "mix.q", m["heads"] * m["dim"], width, 1.5 * sharp)
            if "kv_from" not in m:
                lin(p + "mix.k", m["kv_heads"] * m["dim"], width, 1.5 * sharp)
                lin(p + "mix.v", m["kv_heads"] * m["vdim"], width)
            vec(p + "mix.pb", m["heads"], -2.5, 0.7)
            w[p + "mix.talk"] = bf16_round(np.eye(m["heads"]) + rng.standard_normal((m["heads"], m["heads"])) * 0.4)
            lin(p + "mix.o", width, m["heads"] * m["vdim"], 0.7)
        else:
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for x, n in (("q", nk), ("k", nk), ("v", nv), ("g", nv), ("a1", rank)):
                lin(p + "mix." + x, n, width)
            lin(p + "mix.a2", nk, rank)
            vec(p + "mix.a2.b", nk, 1.5, 1.5)
            vec(p + "mix.norm", m["vdim"], 1.0, 0.2)
            lin(p + "mix.o", width, nv)
        lin(p + "rg1", width, width)
        vec(p + "rg1.b", width, 0.3, 0.7)
        if l["mlp"]:
            r, ff = l["mlp"]["router"], l["mlp"]["expert"]["ff"]
            n = r["experts"] + r.get("identity", 0)
            vec(p + "norm2", width, 1.0, 0.2)
            lin(p + "rg2", width, width)
            vec(p + "rg2.b", width, 0.3, 0.7)
            lin(p + "mlp.router", n, width, 1.5)
            vec(p + "mlp.correction", n, -0.5, 0.1)         # choice scores below zero
            for e in range(r["experts"]):
                lin(f"{p}mlp.e{e}.gate", ff, width, 1.5)
                lin(f"{p}mlp.e{e}.up", ff, width, 1.5)
                lin(f"{p}mlp.e{e}.down", width, ff)
    vec("final.norm", width, 1.0, 0.2)
    lin("head", cfg["vocab"], width)
    return w


def prompts(cfg, lengths, seed=5):
    rng = np.random.default_rng(seed)
    return [list(map(int, rng.integers(0, cfg["vocab"], n))) for n in lengths]


def oracle_logits(cfg, w, ids):
    return fopinex.Model(cfg, w).forward(ids)

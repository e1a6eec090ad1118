"""GPU: the Fopinex mechanisms one at a time through their operators (tm_chunk_attention, tm_gated_linear, tm_moe), against
oracle/fopinex.py.  Inputs are made so that a fault shows: one key stands out, a far token is asked for, experts get
everything or nothing."""
import ctypes as C

import numpy as np
import pytest
import torch

from oracle import fopinex
from tests.test_gpu_rumazen_mechanisms import as_held, pad8, tdtype

pytestmark = pytest.mark.gpu
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


class Attention:
    def __init__(self, dtype, heads, kv, dim, vdim, scale=1.0, size=0, context=512, portion=512, bias=-2.0, seed=0, tiles=0):
        from lmdeploy_b200 import lib as l
        self.l, self.dtype, self.td = l, dtype, tdtype(dtype)
        self.heads, self.kv, self.dim, self.vdim, self.size, self.scale, self.context = heads, kv, dim, vdim, size, scale, context
        es = 4 if dtype == "float32" else 2
        rng = np.random.default_rng(seed)
        self.bias = (bias + 0.5 * rng.standard_normal(heads)).astype(np.float32)
        self.talk = as_held(np.eye(heads) + 0.5 * rng.standard_normal((heads, heads)), "bfloat16").astype(np.float32)
        self.dev = [torch.from_numpy(x).cuda() for x in (self.bias, self.talk)]
        p = self.p = l.TmChunkAttentionParams()
        p.heads, p.kv_heads, p.dim, p.vdim, p.scale, p.chunk = heads, kv, dim, vdim, scale, size
        p.bias, p.talk = (t.data_ptr() for t in self.dev)
        p.ring = -(-(min(context, size + portion) if size else context) // 128) * 128
        p.k_off, p.v_off = 0, -(-kv * p.ring * dim * es // 256) * 256
        self.bytes = p.v_off + kv * p.ring * vdim * es + 256
        p.q_col, p.k_col = 0, pad8(heads * dim)
        p.v_col = p.k_col + pad8(kv * dim)
        p.query_tiles = tiles
        self.ld = p.v_col + pad8(kv * vdim)
        self.out_ld = pad8(heads * vdim)

    def slab(self):
        return torch.full((self.bytes,), 0x3e, dtype=torch.uint8, device="cuda")

    def __call__(self, spans, decode=False, reads_only=False, size=None):
        """spans: list of (slab, history, q, k, v) with rows of the new tokens; -> list of outputs [n, heads, vdim]"""
        n = [s[2].shape[0] for s in spans]
        proj = torch.full((sum(n), self.ld), 3.0, dtype=self.td)
        at = 0
        for (_, _, q, k, v), m in zip(spans, n):
            for col, x in ((self.p.q_col, q), (self.p.k_col, k), (self.p.v_col, v)):
                if x is not None:
                    x = torch.from_numpy(np.ascontiguousarray(np.asarray(x, np.float32).reshape(m, -1)))
                    proj[at:at + m, col:col + x.shape[1]] = x.to(self.td)
            at += m
        proj = proj.cuda()
        out = torch.full((sum(n), self.out_ld), 7.0, dtype=self.td, device="cuda")
        c = self.l.TmMixerCall()
        c.proj, c.proj_ld, c.out, c.out_ld, c.batch = proj.data_ptr(), self.ld, out.data_ptr(), self.out_ld, len(spans)
        c.history, c.n = (C.c_int * len(n))(*[s[1] for s in spans]), (C.c_int * len(n))(*n)
        c.slabs = (C.c_void_p * len(n))(*[s[0].data_ptr() for s in spans])
        c.dtype, c.decode = (1 if self.dtype == "float32" else 0), int(decode)
        self.p.reads_only, self.p.chunk = int(reads_only), self.size if size is None else size
        h, s = self.l.default_handle(0), torch.cuda.current_stream().cuda_stream
        self.l.check(self.l.lib.tm_chunk_attention(h.ptr, C.byref(self.p), C.byref(c), s), "tm_chunk_attention")
        h.check_device_status(s)
        o = out.double().cpu().numpy()[:, :self.heads * self.vdim].reshape(-1, self.heads, self.vdim)
        return np.split(o, np.cumsum(n)[:-1])

    def oracle(self, q, k, v, size=None):
        q, k, v = (as_held(x, self.dtype) for x in (q, k, v))
        return fopinex.mixed_sigmoid_attention(q, k, v, self.scale, self.bias.astype(np.float64), self.talk.astype(np.float64),
                                               self.size if size is None else size)


def worst(got, want, spread=None):
    """largest error over the spread of the wanted values and the value itself (16-bit outputs are rounded)"""
    return (np.abs(got - want) / ((np.std(want) if spread is None else spread) + np.abs(want))).max()


TOL = dict(float32=2e-5, bfloat16=2.5e-2)
SHAPES = [dict(heads=6, kv=2, dim=20, vdim=12, scale=0.3, size=13),
          dict(heads=6, kv=3, dim=64, vdim=64, scale=0.11, size=40),
          dict(heads=8, kv=2, dim=128, vdim=128, scale=0.1, size=129),
          dict(heads=2, kv=2, dim=64, vdim=128, scale=0.2, size=100),
          dict(heads=3, kv=3, dim=33, vdim=70, scale=0.2),
          dict(heads=32, kv=8, dim=128, vdim=64, scale=0.1, size=64),
          dict(heads=40, kv=2, dim=24, vdim=72, scale=0.2, size=21),
          dict(heads=64, kv=16, dim=16, vdim=8, scale=0.3, size=90),
          dict(heads=18, kv=1, dim=64, vdim=64, scale=0.2),
          dict(heads=1, kv=1, dim=8, vdim=8, scale=0.5, size=1),
          dict(heads=12, kv=12, dim=8, vdim=128, scale=0.5, size=50),
          dict(heads=20, kv=20, dim=32, vdim=32, scale=0.3, size=33)]


def random_inputs(a, n, seed=0):
    rng = np.random.default_rng(seed)
    return rng.standard_normal((n, a.heads, a.dim)), rng.standard_normal((n, a.kv, a.dim)), rng.standard_normal((n, a.kv, a.vdim))


def run_in(a, x, sizes, slab=None):
    """the tokens of x in portions of the given sizes (cycled); portions of one token as decode steps"""
    slab, out, at, i = a.slab() if slab is None else slab, [], 0, 0
    while at < len(x[0]):
        n = min(sizes[i % len(sizes)], len(x[0]) - at)
        out += a([(slab, at) + tuple(y[at:at + n] for y in x)], decode=n == 1)
        at, i = at + n, i + 1
    return np.concatenate(out)


@both
@pytest.mark.parametrize("shape", SHAPES, ids=range(len(SHAPES)))
def test_chunk_attention_whole_portions_and_decoding(dtype, shape):
    a = Attention(dtype, **shape)
    x = random_inputs(a, 200)
    want = a.oracle(*x)
    for sizes in ((200,), (2, 3, 1), (64, 1, 7), (129,)):
        got = run_in(a, x, sizes)
        assert worst(got, want) <= TOL[dtype], (sizes, worst(got, want), np.abs(got - want).max((1, 2)).argmax())


@both
@pytest.mark.parametrize("bias", [-15.0, 6.0])
def test_weights_that_are_tiny_or_all_but_one(dtype, bias):
    a = Attention(dtype, 8, 2, 64, 64, scale=0.1, size=90, bias=bias)
    x = random_inputs(a, 150)
    want = a.oracle(*x)
    for sizes in ((150,), (40, 1, 1)):
        assert worst(run_in(a, x, sizes), want) <= TOL[dtype], sizes


@both
@pytest.mark.parametrize("dims", [(16, 16), (64, 64), (128, 128), (20, 12)])
@pytest.mark.parametrize("size", [1, 32, 100, 130, 0])
def test_one_key_stands_out_on_either_side_of_every_edge(dtype, dims, size):
    """The queries look for one direction only, and one token's key has it: its value tells whether it is seen, up to the end
    of its chunk and not beyond."""
    n = 300
    a = Attention(dtype, 3, 1, *dims, scale=1.0, size=size, context=n, bias=-12.0, tiles=1)
    edge = size or 128
    rng = np.random.default_rng(1)
    for spot in sorted({0, 1, edge - 1, edge, edge + 1, 2 * edge - 1, 63, 64, 127, 128, n - 2} & set(range(n))):
        q = np.zeros((n, 3, dims[0]))
        q[:, 0, 0], q[:, 1, 1], q[:, 2, 0] = 5.0, 5.0, -5.0
        k = rng.standard_normal((n, 1, dims[0])) * 0.05
        k[spot, 0, 0] = 6.0                       # score 30 for head 0 only
        v = rng.standard_normal((n, 1, dims[1])) * 0.1
        v[spot] += 3.0
        want = a.oracle(q, k, v)
        last = min(n, (spot // size + 1) * size if size else n)
        own = want.mean(2) @ np.linalg.pinv(a.talk.astype(np.float64).T)      # back from the mixed heads to head 0
        assert own[spot:last, 0].min() > 1.0 and (last == n or np.abs(own[last:, 0]).max() < 0.1)
        got = run_in(a, (q, k, v), (n,))
        assert np.abs(got - want).max() <= 3 * TOL[dtype], (spot, "prompt", np.abs(got - want).max((1, 2)).argmax())
        # decoding across the end of the chunk
        slab, at = a.slab(), 0
        for p in sorted({spot + 1, last} & set(range(3, n - 3))):
            if p - 2 > at:
                a([(slab, at, q[at:p - 2], k[at:p - 2], v[at:p - 2])])
                at = p - 2
            while at < min(p + 3, n):
                got = a([(slab, at, q[at:at + 1], k[at:at + 1], v[at:at + 1])], decode=True)[0]
                assert np.abs(got[0] - want[at]).max() <= 3 * TOL[dtype], (spot, "decoded", at)
                at += 1


@both
@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[1], SHAPES[2], SHAPES[6], SHAPES[7], SHAPES[9]], ids=range(6))
def test_chunk_attention_in_a_short_ring_and_unequal_batches(dtype, shape):
    """token rows wrap around many times; sequences of different lengths share every launch"""
    a = Attention(dtype, context=700, portion=40, tiles=2, **shape)
    assert a.p.ring < 500
    lens = (600, 31, 257)
    x = [random_inputs(a, n, 10 + i) for i, n in enumerate(lens)]
    want, slabs, at, step = [a.oracle(*y) for y in x], [a.slab() for _ in lens], [0] * len(lens), 0
    while any(p < n for p, n in zip(at, lens)):
        live = [i for i in range(len(lens)) if at[i] < lens[i]]
        decode = step % 4 == 3
        n = {i: 1 if decode else min(1 + (17 * step + 13 * i) % 40, lens[i] - at[i]) for i in live}
        got = a([(slabs[i], at[i]) + tuple(y[at[i]:at[i] + n[i]] for y in x[i]) for i in live], decode=decode)
        for i, o in zip(live, got):
            assert worst(o, want[i][at[i]:at[i] + n[i]], np.std(want[i])) <= TOL[dtype], (i, at[i], n[i])
            at[i] += n[i]
        step += 1


@both
@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[1], SHAPES[2], SHAPES[4], SHAPES[11]], ids=range(5))
def test_keys_and_values_of_another_layer(dtype, shape):
    """a reader sees what the writer cached, with queries and a chunk of its own, in prompts and while decoding"""
    a = Attention(dtype, context=400, **shape)
    other = 3 * (shape.get("size") or 20) // 2
    a.p.ring = max(a.p.ring, 512)
    es = 4 if dtype == "float32" else 2
    a.p.v_off = a.kv * a.p.ring * a.dim * es
    a.bytes = a.p.v_off + a.kv * a.p.ring * a.vdim * es
    q, k, v = random_inputs(a, 150)
    q2 = random_inputs(a, 150, 7)[0]
    want, want2 = a.oracle(q, k, v), a.oracle(q2, k, v, other)
    slab, at = a.slab(), 0
    for n in (70, 2, 1, 1, 1, 40, 1, 1, 33):
        before = slab.clone() if at else None
        got = a([(slab, at, q[at:at + n], k[at:at + n], v[at:at + n])], decode=n == 1)[0]
        held = slab.clone()
        got2 = a([(slab, at, q2[at:at + n], None, None)], decode=n == 1, reads_only=True, size=other)[0]
        assert torch.equal(held, slab) and (before is None or not torch.equal(before, held))
        assert worst(got, want[at:at + n], np.std(want)) <= TOL[dtype], (at, "own")
        assert worst(got2, want2[at:at + n], np.std(want2)) <= TOL[dtype], (at, "shared")
        at += n


def test_chunk_attention_refuses_what_does_not_fit():
    from lmdeploy_b200 import lib as l
    a = Attention("float32", 2, 1, 16, 16, size=8, context=64, portion=64)
    with pytest.raises(l.TmError):
        a([(a.slab(), 0) + random_inputs(a, 200)])          # more tokens than the ring holds
    b = Attention("float32", 2, 2, 300, 16)
    with pytest.raises(l.TmError):
        b([(b.slab(), 0) + random_inputs(b, 4)])            # heads larger than the kernels take


class Linear:
    def __init__(self, dtype, heads, dim, vdim, rank, tau, seed=0, eps=1e-4):
        from lmdeploy_b200 import lib as l
        self.l, self.dtype, self.td, self.heads, self.dim, self.vdim, self.rank, self.tau, self.eps = \
            l, dtype, tdtype(dtype), heads, dim, vdim, rank, tau, eps
        rng, n, nv = np.random.default_rng(seed), heads * dim, heads * vdim
        self.w2 = as_held(rng.standard_normal((n, rank)), dtype)
        self.bias, self.norm = rng.standard_normal(n) * 3, 1 + 0.2 * rng.standard_normal(vdim)
        self.w2_ld = pad8(rank)
        w2 = torch.zeros(n, self.w2_ld, dtype=self.td)
        w2[:, :rank] = torch.from_numpy(self.w2).to(self.td)
        self.dev = [w2.cuda()] + [torch.from_numpy(v).float().cuda() for v in (self.bias, self.norm)]
        p = self.p = l.TmGatedLinearParams()
        p.heads, p.dim, p.vdim, p.rank, p.w2, p.w2_ld = heads, dim, vdim, rank, self.dev[0].data_ptr(), self.w2_ld
        p.bias, p.norm = (t.data_ptr() for t in self.dev[1:])
        p.norm_eps, p.scale, p.tau, p.state_off = eps, dim ** -0.5, tau, 256
        self.cols, at = {}, 0
        for name, m in (("q", n), ("k", n), ("v", nv), ("g", nv), ("a", rank)):
            setattr(p, name + "_col", at)
            self.cols[name] = (at, m)
            at += pad8(m)
        self.ld, self.out_ld = at, pad8(nv)

    def slab(self):
        return torch.full((256 + self.heads * self.dim * self.vdim * 4,), 0x3e, dtype=torch.uint8, device="cuda")

    def __call__(self, spans, decode=False):
        n = [len(s[2]["q"]) for s in spans]
        proj = torch.zeros(sum(n), self.ld, dtype=self.td)
        at = 0
        for (_, _, x), m in zip(spans, n):
            for name, (col, w) in self.cols.items():
                proj[at:at + m, col:col + w] = torch.from_numpy(np.ascontiguousarray(x[name])).to(self.td)
            at += m
        proj, out = proj.cuda(), torch.full((sum(n), self.out_ld), 7.0, dtype=self.td, device="cuda")
        c = self.l.TmMixerCall()
        c.proj, c.proj_ld, c.out, c.out_ld, c.batch = proj.data_ptr(), self.ld, out.data_ptr(), self.out_ld, len(spans)
        c.history, c.n = (C.c_int * len(n))(*[s[1] for s in spans]), (C.c_int * len(n))(*n)
        c.slabs = (C.c_void_p * len(n))(*[s[0].data_ptr() for s in spans])
        c.dtype, c.decode = (1 if self.dtype == "float32" else 0), int(decode)
        h, s = self.l.default_handle(0), torch.cuda.current_stream().cuda_stream
        self.l.check(self.l.lib.tm_gated_linear(h.ptr, C.byref(self.p), C.byref(c), s), "tm_gated_linear")
        h.check_device_status(s)
        return np.split(out.double().cpu().numpy()[:, :self.heads * self.vdim], np.cumsum(n)[:-1])

    def inputs(self, n, seed):
        rng = np.random.default_rng(seed)
        return {name: rng.standard_normal((n, w)) for name, (_, w) in self.cols.items()}

    def oracle(self, x):
        x = {k: as_held(v, self.dtype) for k, v in x.items()}
        n, f32 = len(x["q"]), lambda v: v.astype(np.float32).astype(np.float64)
        key, val = (n, self.heads, self.dim), (n, self.heads, self.vdim)
        decay = fopinex.gla_decay(x["a"] @ self.w2.T + f32(self.bias), self.tau).reshape(key)
        o, s = fopinex.gated_linear_attention(x["q"].reshape(key) * self.dim ** -0.5, x["k"].reshape(key), x["v"].reshape(val), decay,
                                              np.zeros((self.heads, self.dim, self.vdim)))
        return fopinex.rms_norm(o, f32(self.norm), self.eps).reshape(n, -1) * x["g"] * fopinex.sigmoid(x["g"]), s

    def feed(self, slab, x, sizes):
        got, at, i = [], 0, 0
        while at < len(x["q"]):
            m = min(sizes[i % len(sizes)], len(x["q"]) - at)
            got += self([(slab, at, {k: v[at:at + m] for k, v in x.items()})], decode=m == 1)
            at, i = at + m, i + 1
        return np.concatenate(got)


LINEAR = [(3, 64, 64, 32, 16.0), (2, 128, 128, 16, 4.0), (5, 24, 40, 7, 1.0), (1, 1, 1, 1, 1.0), (2, 16, 200, 3, 9.0), (4, 32, 16, 64, 0.5),
          (1, 200, 12, 12, 16.0), (2, 65, 9, 9, 30.0), (2, 48, 64, 130, 2.0), (2, 256, 256, 8, 16.0)]


@both
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", LINEAR)
def test_gated_linear_whole_portions_and_decoding(dtype, heads, dim, vdim, rank, tau):
    d = Linear(dtype, heads, dim, vdim, rank, tau)
    n = 75
    x = d.inputs(n, 3)
    want, state = d.oracle(x)
    tol = 2e-4 if dtype == "float32" else 4e-2
    for sizes in ((n,), (2,), (1,), (17, 1, 3), (16,), (33,)):
        slab = d.slab()
        got = d.feed(slab, x, sizes)
        assert np.abs(got - want).max() <= tol, (sizes, np.abs(got - want).max())
        # the state is fp32 in both precisions, and exact to fp32
        held = slab[256:].view(torch.float32).cpu().numpy().reshape(heads, vdim, dim).transpose(0, 2, 1)
        assert np.abs(held - state).max() <= 2e-5 * np.abs(state).max(), sizes


@both
def test_gated_linear_remembers_a_far_token_and_forgets_where_the_decay_says_so(dtype):
    """one key channel that keeps everything, one that decays fast: the first token's value comes back hundreds of tokens
    later along the one, and not along the other"""
    d = Linear(dtype, 2, 64, 48, 4, 16.0)
    n = 500
    x = {k: np.zeros_like(v) for k, v in d.inputs(n, 0).items()}
    d.bias[:], d.bias[7::64] = 20.0, -3.0
    d.dev[1].copy_(torch.from_numpy(d.bias).float())
    value = as_held(np.random.default_rng(4).standard_normal(48), dtype)
    x["k"][:, 1::64] = 1.0                        # every token writes zero along one key direction ...
    x["k"][0], x["v"][0] = 0.0, np.tile(value, 2)
    x["k"][0, 5::64] = x["k"][0, 7::64] = 1.0     # ... except the first, along two others
    x["v"][1:] = np.random.default_rng(5).standard_normal((n - 1, 96)) * 0.1
    x["q"][:, 5::64] = 8.0
    x["q"][n // 2:, 7::64], x["q"][n // 2:, 5::64] = 8.0, 0.0
    x["q"][-1, 5::64], x["q"][-1, 7::64] = 8.0, 0.0
    x["g"][:] = 1.0
    want, _ = d.oracle(x)
    value_out = np.tile(value / np.sqrt((value ** 2).mean()) * d.norm.astype(np.float32), 2) * fopinex.sigmoid(1.0)
    assert np.abs(want[-1] - value_out).max() < 1e-2 and np.abs(want[-2]).max() < 0.2 * np.abs(value_out).max()
    slab = d.slab()
    got = d.feed(slab, {k: v[:490] for k, v in x.items()}, (490,))
    assert np.abs(got - want[:490]).max() <= (1e-3 if dtype == "float32" else 4e-2)
    for t in range(490, n):
        got = d([(slab, t, {k: v[t:t + 1] for k, v in x.items()})], decode=True)[0]
    assert np.abs(got[0] - want[-1]).max() <= (1e-3 if dtype == "float32" else 4e-2)


@both
def test_gated_linear_unequal_batches(dtype):
    d = Linear(dtype, 3, 48, 56, 5, 8.0)
    lens = (90, 7, 33, 1)
    x = [d.inputs(n, 20 + i) for i, n in enumerate(lens)]
    want, slabs, at, step = [d.oracle(y)[0] for y in x], [d.slab() for _ in lens], [0] * 4, 0
    tol = 2e-4 if dtype == "float32" else 4e-2
    while any(p < n for p, n in zip(at, lens)):
        live = [i for i in range(4) if at[i] < lens[i]]
        decode = step % 3 == 2
        n = {i: 1 if decode else min(1 + (11 * step + 7 * i) % 23, lens[i] - at[i]) for i in live}
        got = d([(slabs[i], at[i], {k: v[at[i]:at[i] + n[i]] for k, v in x[i].items()}) for i in live], decode=decode)
        for i, o in zip(live, got):
            assert np.abs(o - want[i][at[i]:at[i] + n[i]]).max() <= tol, (i, at[i])
            at[i] += n[i]
        step += 1


def run_moe(dtype, tokens, width, ff, experts, identity, top, groups=1, keep=1, limit=1.1, logits=None, seed=0, correction=None):
    """-> (x, norm of x, wanted x)"""
    from lmdeploy_b200 import lib as l
    rng, td, n = np.random.default_rng(seed), tdtype(dtype), experts + identity
    ld, fld = pad8(width), pad8(ff)
    held = lambda x: as_held(x, dtype)
    h, gate = held(rng.standard_normal((tokens, width))), held(rng.standard_normal((tokens, width)))
    wg, wu = (held(rng.standard_normal((experts, ff, width)) * 1.5 / np.sqrt(width)) for _ in range(2))
    wd = held(rng.standard_normal((experts, width, ff)) / np.sqrt(ff))
    x0 = rng.standard_normal((tokens, width)).astype(np.float32)
    z = rng.standard_normal((tokens, n)).astype(np.float32) * 2 if logits is None else np.asarray(logits, np.float32)
    corr = (rng.standard_normal(n) * 0.1 - 0.6).astype(np.float32) if correction is None else np.asarray(correction, np.float32)
    gb, nw = rng.standard_normal(width).astype(np.float32), rng.standard_normal(width).astype(np.float32)

    def dev(a, ld_):
        t = torch.full(a.shape[:-1] + (ld_,), float("nan"), dtype=td)
        t[..., :a.shape[-1]] = torch.from_numpy(a).to(td)
        return t.cuda()
    we = np.empty((experts, 2 * ff, width))
    we[:, 0::2], we[:, 1::2] = wg, wu
    t_h, t_gate, t_we, t_wd = dev(h, ld), dev(gate, ld), dev(we, ld), dev(wd, fld)
    t_x, t_z = torch.from_numpy(x0).cuda(), torch.from_numpy(np.pad(z, ((0, 0), (0, 3)), constant_values=np.nan)).cuda()
    vecs = [torch.from_numpy(v).cuda() for v in (gb, corr, nw)]
    out = torch.full((tokens, ld), 9.0, dtype=td, device="cuda")
    p = l.TmMoeParams()
    p.tokens, p.width, p.ff, p.experts, p.identity, p.top, p.groups, p.keep = tokens, width, ff, experts, identity, top, groups, keep
    p.limit, p.slope, p.mult, p.norm_eps = limit, 1.702, 0.7, 1e-3
    p.x, p.logits, p.logits_ld, p.input, p.input_ld, p.gate, p.gate_ld = t_x.data_ptr(), t_z.data_ptr(), n + 3, t_h.data_ptr(), ld, t_gate.data_ptr(), ld
    p.gate_bias, p.correction, p.norm_weight = (v.data_ptr() for v in vecs)
    p.w_experts, p.w_down, p.norm_out, p.dtype = t_we.data_ptr(), t_wd.data_ptr(), out.data_ptr(), int(dtype == "float32")
    hd, s = l.default_handle(0), torch.cuda.current_stream().cuda_stream
    l.check(l.lib.tm_moe(hd.ptr, C.byref(p), s), "tm_moe")
    hd.check_device_status(s)
    want = np.zeros((tokens, width))
    for t in range(tokens):
        for e, sc in zip(*fopinex.route(z[t].astype(np.float64), corr.astype(np.float64), top, groups, keep)):
            want[t] += sc * (fopinex.clamped_expert(h[t], wg[e], wu[e], wd[e], limit) if e < experts else h[t])
    want = x0 + 0.7 * fopinex.sigmoid(gate + gb) * want
    return t_x.double().cpu().numpy(), out.double().cpu().numpy()[:, :width], want, fopinex.rms_norm(want, nw.astype(np.float64), 1e-3)


MOE = [dict(width=40, ff=24, experts=5, identity=3, top=3, groups=4, keep=2), dict(width=256, ff=128, experts=16, identity=0, top=4),
       dict(width=151, ff=65, experts=33, identity=7, top=6, groups=8, keep=3), dict(width=16, ff=1, experts=1, identity=0, top=1),
       dict(width=72, ff=200, experts=1, identity=1, top=2), dict(width=64, ff=64, experts=2, identity=30, top=8, groups=16, keep=4),
       dict(width=136, ff=72, experts=130, identity=2, top=12, groups=3, keep=1)]


@both
@pytest.mark.parametrize("shape", MOE, ids=range(len(MOE)))
@pytest.mark.parametrize("tokens", [1, 2, 8, 9, 64, 190])
def test_mixture_of_experts(dtype, shape, tokens):
    x, norm, want, want_norm = run_moe(dtype, tokens, seed=tokens, **shape)
    tol = 3e-5 if dtype == "float32" else 2.5e-2
    assert np.abs(x - want).max() <= tol, np.abs(x - want).max()
    assert np.abs(norm - want_norm).max() <= 3 * tol, np.abs(norm - want_norm).max()


@both
@pytest.mark.parametrize("tokens", [3, 64, 600])
def test_experts_that_get_everything_or_nothing(dtype, tokens):
    rng = np.random.default_rng(2)
    z = rng.standard_normal((tokens, 10)) * 0.1
    z[:, 6] += 4.0                                # everybody's first choice; the second is an identity expert
    z[:, 9] += 2.0
    x, _, want, _ = run_moe(dtype, tokens, 96, 48, 8, 2, 2, logits=z, correction=np.full(10, -1.0))
    assert np.abs(x - want).max() <= (3e-5 if dtype == "float32" else 2.5e-2)
    z[:, 8] += 9.0                                # identity experts only: no expert has a row
    x, _, want, _ = run_moe(dtype, tokens, 96, 48, 8, 2, 2, logits=z, correction=np.full(10, -1.0))
    assert np.abs(x - want).max() <= (3e-5 if dtype == "float32" else 2.5e-2)


def test_choice_is_by_corrected_scores_within_the_best_groups_and_weights_are_not():
    """a correction that lifts a poor expert: chosen, but weighted by its poor score; a group left out although it holds the
    second best expert"""
    z = np.log(np.array([[0.40, 0.05, 0.30, 0.02, 0.13, 0.10]]))
    corr = np.array([-1.0, -1.0, -1.0, -0.2, -1.0, -1.0])       # choice: -.6 -.95 | -.7 -.18 | -.87 -.9
    chosen, s = fopinex.route(z[0], corr, 2, 3, 1)
    assert chosen == [3, 2] and np.allclose(s, [0.02, 0.30])
    x, _, want, _ = run_moe("float32", 1, 32, 16, 5, 1, 2, 3, 1, logits=z, correction=corr)
    assert np.abs(x - want).max() <= 3e-5
    x, _, want, _ = run_moe("float32", 1, 32, 16, 5, 1, 3, 3, 2, logits=z, correction=corr)
    assert np.abs(x - want).max() <= 3e-5

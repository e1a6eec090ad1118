"""GPU: the Rumazen mechanisms one at a time through their operators (tm_window_attention, tm_delta_rule, tm_gemm_dense),
against oracle/rumazen.py.  Inputs are made so that a fault shows: one score stands out, at a chosen distance."""
import ctypes as C

import numpy as np
import pytest
import torch

from oracle import rumazen

pytestmark = pytest.mark.gpu


def tdtype(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def as_held(x, dtype):
    return torch.from_numpy(np.asarray(x, np.float32)).to(tdtype(dtype)).double().numpy()


def pad8(n):
    return (n + 7) // 8 * 8


class Attention:
    def __init__(self, dtype, heads, kv, dim, vdim, rot=0, base=100.0, factor=1.0, scale=1.0, softcap=0.0, size=0, pool=0, context=512, portion=512):
        from lmdeploy_b200 import lib as l
        self.l, self.dtype, self.td = l, dtype, tdtype(dtype)
        self.heads, self.kv, self.dim, self.vdim, self.size, self.pool = heads, kv, dim, vdim, size, pool
        self.rot, self.base, self.factor, self.scale, self.softcap = rot, base, factor, scale, softcap
        es = 4 if dtype == "float32" else 2
        p = self.p = l.TmWindowAttentionParams()
        p.heads, p.kv_heads, p.dim, p.vdim, p.rot_dims = heads, kv, dim, vdim, rot
        self.freq = torch.tensor([base ** (-2.0 * i / rot) / factor for i in range(rot // 2)] or [0.0], dtype=torch.float64).float().cuda()
        p.inv_freq, p.scale, p.softcap, p.window, p.pool = self.freq.data_ptr(), scale, softcap, size, pool
        p.ring = -(-(min(context, max(size, pool) + portion) if size else context) // 128) * 128
        p.pool_rows = context // pool + 1 if pool else 0
        at = 0
        for name, n in (("k_off", p.ring * dim), ("v_off", p.ring * vdim), ("pooled_k_off", p.pool_rows * dim), ("pooled_v_off", p.pool_rows * vdim)):
            setattr(p, name, at)
            at += -(-kv * n * es // 256) * 256
        self.bytes = at + 256
        p.q_col, p.k_col = 0, pad8(heads * dim)
        p.v_col = p.k_col + pad8(kv * dim)
        p.g_col = p.v_col + pad8(kv * vdim)
        self.ld = p.g_col + pad8(heads)
        self.out_ld = pad8(heads * vdim)

    def slab(self):
        return torch.full((self.bytes,), 0x3e, dtype=torch.uint8, device="cuda")

    def __call__(self, spans, decode=False):
        """spans: list of (slab, history, q, k, v, g) with rows of the new tokens; -> list of outputs [n, heads, vdim]"""
        n = [s[2].shape[0] for s in spans]
        proj = torch.zeros(sum(n), self.ld, dtype=self.td)
        at = 0
        for (_, _, q, k, v, g), m in zip(spans, n):
            for col, x in ((self.p.q_col, q), (self.p.k_col, k), (self.p.v_col, v), (self.p.g_col, g)):
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
        h = self.l.default_handle(0)
        self.l.check(self.l.lib.tm_window_attention(h.ptr, C.byref(self.p), C.byref(c), torch.cuda.current_stream().cuda_stream), "tm_window_attention")
        h.check_device_status(torch.cuda.current_stream().cuda_stream)
        o = out.double().cpu().numpy()[:, :self.heads * self.vdim].reshape(-1, self.heads, self.vdim)
        return np.split(o, np.cumsum(n)[:-1])

    def oracle(self, q, k, v, g):
        q, k, v, g = (as_held(x, self.dtype) for x in (q, k, v, g))
        pos = np.arange(len(q))
        q = rumazen.rotate_interleaved(q, pos, self.rot, self.base, self.factor)
        k = as_held(rumazen.rotate_interleaved(k, pos, self.rot, self.base, self.factor), self.dtype)
        o = rumazen.window_attention(q, k, v, self.scale, self.size, self.pool, self.softcap)
        return o * rumazen.sigmoid(g)[:, :, None]


TOL = dict(float32=3e-5, bfloat16=2e-2)
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
SHAPES = [dict(heads=6, kv=2, dim=20, vdim=12, rot=12, factor=2.0, scale=0.3, softcap=4.0, size=13, pool=3),
          dict(heads=6, kv=3, dim=64, vdim=64, rot=64, base=5000.0, scale=0.11, softcap=22.0, size=40, pool=9),
          dict(heads=8, kv=2, dim=128, vdim=128, rot=64, base=300.0, factor=4.0, scale=0.1, softcap=12.0, size=129, pool=16),
          dict(heads=2, kv=2, dim=64, vdim=128, scale=0.2, size=100),
          dict(heads=3, kv=3, dim=33, vdim=70, rot=32, scale=0.2, softcap=2.0),
          dict(heads=2, kv=1, dim=128, vdim=64, rot=16, scale=0.1, softcap=50.0, size=7, pool=64),
          dict(heads=40, kv=2, dim=24, vdim=72, rot=24, scale=0.2, softcap=70.0, size=21, pool=6),
          dict(heads=16, kv=1, dim=64, vdim=64, rot=2, scale=0.2, softcap=8.0, size=1, pool=1)]


def random_inputs(a, n, seed=0):
    rng = np.random.default_rng(seed)
    return (rng.standard_normal((n, a.heads, a.dim)), rng.standard_normal((n, a.kv, a.dim)), rng.standard_normal((n, a.kv, a.vdim)),
            rng.standard_normal((n, a.heads)))


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
def test_window_attention_whole_portions_and_decoding(dtype, shape):
    a = Attention(dtype, **shape)
    x = random_inputs(a, 200)
    want = a.oracle(*x)
    for sizes in ((200,), (2, 3, 1), (64, 1, 7), (129,)):
        got = run_in(a, x, sizes)
        assert np.abs(got - want).max() <= TOL[dtype], (sizes, np.abs(got - want).max(), np.abs(got - want).max((1, 2)).argmax())


@both
@pytest.mark.parametrize("dims", [(16, 16), (64, 64), (128, 128)])
@pytest.mark.parametrize("size,pool", [(32, 4), (100, 16), (130, 128), (3, 1)])
def test_one_key_stands_out_at_every_edge(dtype, dims, size, pool):
    """The queries look for one direction only, and one token's key has it: its value tells whether (and with which weight)
    it is seen — as a token just inside the window, as nothing just outside, as part of a block as soon as the block has
    left, and far away."""
    n = 300
    a = Attention(dtype, 2, 1, *dims, scale=1.0, softcap=25.0, size=size, pool=pool, context=n)
    rng = np.random.default_rng(1)
    spots = sorted({0, 1, pool - 1, pool, 63, 64, 127, 128, n - size - 1, n - size, n - size + 1, n - size - pool, n - 2} & set(range(n)))
    for spot in spots:
        q = np.zeros((n, 2, dims[0]))
        q[:, 0, 0], q[:, 1, 1] = 5.0, 5.0
        k = rng.standard_normal((n, 1, dims[0])) * 0.05
        k[spot, 0, 0] = 4.0                      # score 20 for head 0 only; a block of it scores 20 / pool
        v = rng.standard_normal((n, 1, dims[1])) * 0.1
        v[spot] += 3.0
        x = (q, k, v, np.zeros((n, 2)))
        want = a.oracle(*x)
        first = spot + size                       # the first position that no longer sees it as a token
        if first < n and pool > 1:
            assert want[first - 1, 0].mean() > 1.2 and want[first, 0].mean() < 1.0
        got = run_in(a, x, (n,))
        assert np.abs(got - want).max() <= 2 * TOL[dtype], (spot, "prompt", np.abs(got - want).max((1, 2)).argmax())
        # decoding across the edges: the window's, and the block's
        slab = a.slab()
        edges = [p for p in (first, (spot // pool + 1) * pool - 1 + size) if 2 < p < n - 3]
        at = 0
        for p in sorted(set(edges)):
            if p - 2 > at:
                a([(slab, at) + tuple(y[at:p - 2] for y in x)])
                at = p - 2
            while at < min(p + 3, n):
                got = a([(slab, at) + tuple(y[at:at + 1] for y in x)], decode=True)[0]
                assert np.abs(got[0] - want[at]).max() <= 2 * TOL[dtype], (spot, "decoded", at)
                at += 1


@both
@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[1], SHAPES[2], SHAPES[6], SHAPES[7]], ids=range(5))
def test_window_attention_in_a_short_ring_and_unequal_batches(dtype, shape):
    """token rows wrap around many times; sequences of different lengths share every launch"""
    a = Attention(dtype, context=700, portion=40, **shape)
    assert a.p.ring < 500
    lens = (600, 31, 257)
    x = [random_inputs(a, n, 10 + i) for i, n in enumerate(lens)]
    want, slabs, at = [a.oracle(*y) for y in x], [a.slab() for _ in lens], [0] * len(lens)
    step = 0
    while any(p < n for p, n in zip(at, lens)):
        live = [i for i in range(len(lens)) if at[i] < lens[i]]
        decode = step % 4 == 3
        n = {i: 1 if decode else min(1 + (17 * step + 13 * i) % 40, lens[i] - at[i]) for i in live}
        got = a([(slabs[i], at[i]) + tuple(y[at[i]:at[i] + n[i]] for y in x[i]) for i in live], decode=decode)
        for i, o in zip(live, got):
            assert np.abs(o - want[i][at[i]:at[i] + n[i]]).max() <= TOL[dtype], (i, at[i], n[i])
            at[i] += n[i]
        step += 1


def test_window_attention_refuses_what_does_not_fit():
    from lmdeploy_b200 import lib as l
    a = Attention("float32", 2, 1, 16, 16, size=8, pool=4, context=64, portion=64)
    x = random_inputs(a, 200)
    with pytest.raises(l.TmError):
        a([(a.slab(), 0) + x])                       # more tokens than the ring holds
    b = Attention("float32", 2, 2, 300, 16)
    with pytest.raises(l.TmError):
        b([(b.slab(), 0) + random_inputs(b, 4)])     # heads larger than the kernels take


class Delta:
    def __init__(self, dtype, heads, dim, rank, seed=0, eps=1e-4):
        from lmdeploy_b200 import lib as l
        self.l, self.dtype, self.td, self.heads, self.dim, self.rank, self.eps = l, dtype, tdtype(dtype), heads, dim, rank, eps
        rng, n = np.random.default_rng(seed), heads * dim
        self.w2 = as_held(rng.standard_normal((n, rank)), dtype)
        self.w0, self.ab, self.norm = rng.standard_normal(n) * 2 - 1, rng.standard_normal(n), 1 + 0.2 * rng.standard_normal(n)
        self.w2_ld = pad8(rank)
        w2 = torch.zeros(n, self.w2_ld, dtype=self.td)
        w2[:, :rank] = torch.from_numpy(self.w2).to(self.td)
        self.dev = [w2.cuda()] + [torch.from_numpy(v).float().cuda() for v in (self.w0, self.ab, self.norm)]
        p = self.p = l.TmDeltaRuleParams()
        p.heads, p.dim, p.rank, p.w2, p.w2_ld = heads, dim, rank, self.dev[0].data_ptr(), self.w2_ld
        p.w0, p.a_bias, p.norm = (t.data_ptr() for t in self.dev[1:])
        p.norm_eps, p.unit_eps, p.decay_scale, p.state_off = eps, 1e-6, float(np.exp(-0.5)), 256
        self.cols = {}
        at = 0
        for name, m in (("r", n), ("k", n), ("v", n), ("a", n), ("g", n), ("w1", rank)):
            setattr(p, name + "_col", at)
            self.cols[name] = (at, m)
            at += pad8(m)
        self.ld, self.out_ld = at, pad8(n)

    def slab(self):
        return torch.full((256 + self.heads * self.dim ** 2 * 4,), 0x3e, dtype=torch.uint8, device="cuda")

    def __call__(self, spans, decode=False):
        n = [len(s[2]["r"]) for s in spans]
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
        h = self.l.default_handle(0)
        self.l.check(self.l.lib.tm_delta_rule(h.ptr, C.byref(self.p), C.byref(c), torch.cuda.current_stream().cuda_stream), "tm_delta_rule")
        h.check_device_status(torch.cuda.current_stream().cuda_stream)
        return np.split(out.double().cpu().numpy()[:, :self.heads * self.dim], np.cumsum(n)[:-1])

    def inputs(self, n, seed, scale=1.0):
        rng = np.random.default_rng(seed)
        x = {name: rng.standard_normal((n, w)) * scale for name, (_, w) in self.cols.items()}
        x["w1"] = np.tanh(x["w1"])
        return x

    def oracle(self, x):
        x = {k: as_held(v, self.dtype) for k, v in x.items()}
        n, shape = len(x["r"]), (len(x["r"]), self.heads, self.dim)
        f32 = lambda v: v.astype(np.float32).astype(np.float64)
        w = rumazen.delta_decay(x["w1"] @ self.w2.T + f32(self.w0)).reshape(shape)
        a = rumazen.sigmoid(x["a"] + f32(self.ab)).reshape(shape)
        o, s = rumazen.delta_rule(x["r"].reshape(shape), x["k"].reshape(shape), x["v"].reshape(shape), w, a,
                                  np.zeros((self.heads, self.dim, self.dim)))
        return rumazen.rms(o, self.eps).reshape(n, -1) * f32(self.norm) * rumazen.sigmoid(x["g"]), s


@both
@pytest.mark.parametrize("heads,dim,rank", [(3, 64, 32), (2, 128, 40), (5, 24, 7), (1, 1, 1), (2, 16, 3), (4, 32, 64), (1, 200, 12), (2, 65, 9)])
def test_delta_rule_whole_portions_and_decoding(dtype, heads, dim, rank):
    d = Delta(dtype, heads, dim, rank)
    n = 75
    x = d.inputs(n, 3)
    want, state = d.oracle(x)
    tol = 2e-4 if dtype == "float32" else 3e-2
    for sizes in ((n,), (2,), (1,), (17, 1, 3), (16,), (33,)):
        slab, got, at, i = d.slab(), [], 0, 0
        while at < n:
            m = min(sizes[i % len(sizes)], n - at)
            got += d([(slab, at, {k: v[at:at + m] for k, v in x.items()})], decode=m == 1)
            at, i = at + m, i + 1
        assert np.abs(np.concatenate(got) - want).max() <= tol, (sizes, np.abs(np.concatenate(got) - want).max())
        # the state is fp32 in both precisions, and exact to fp32
        held = slab[256:].view(torch.float32).cpu().numpy().reshape(state.shape).transpose(0, 2, 1)   # [head][value][key]
        assert np.abs(held - state).max() <= 2e-5 * np.abs(state).max(), sizes


@both
def test_delta_rule_remembers_a_far_token(dtype):
    """decay close to one and nothing removed: the first token's value comes back hundreds of tokens later"""
    d = Delta(dtype, 2, 64, 4)
    n = 400
    x = {k: np.zeros_like(v) for k, v in d.inputs(n, 0).items()}
    d.w0[:] = -14.0
    d.dev[1].copy_(torch.from_numpy(d.w0).float())
    d.ab[:] = -20.0
    d.dev[2].copy_(torch.from_numpy(d.ab).float())
    rng = np.random.default_rng(4)
    value = as_held(rng.standard_normal(64), dtype)
    x["k"][:, 1::64] = 1.0                        # every token writes along one key direction with value zero ...
    x["k"][0], x["v"][0] = 0.0, np.tile(value, 2)
    x["k"][0, 5::64] = 1.0                        # ... except the first, along another
    x["r"][-1, 5::64] = 1.0
    want, _ = d.oracle(x)
    assert np.abs(want[-1] - value_norm(value, d)).max() < 1e-3
    slab = d.slab()
    d([(slab, 0, {k: v[:390] for k, v in x.items()})])
    for t in range(390, n):
        got = d([(slab, t, {k: v[t:t + 1] for k, v in x.items()})], decode=True)[0]
    assert np.abs(got[0] - want[-1]).max() <= (1e-4 if dtype == "float32" else 2e-2)


def value_norm(value, d):
    return np.tile(value / np.sqrt((value ** 2).mean()), 2) * d.norm.astype(np.float32) * 0.5


@both
def test_delta_rule_unequal_batches(dtype):
    d = Delta(dtype, 3, 48, 5)
    lens = (90, 7, 33, 1)
    x = [d.inputs(n, 20 + i) for i, n in enumerate(lens)]
    want, slabs, at, step = [d.oracle(y)[0] for y in x], [d.slab() for _ in lens], [0] * 4, 0
    tol = 2e-4 if dtype == "float32" else 3e-2
    while any(p < n for p, n in zip(at, lens)):
        live = [i for i in range(4) if at[i] < lens[i]]
        decode = step % 3 == 2
        n = {i: 1 if decode else min(1 + (11 * step + 7 * i) % 23, lens[i] - at[i]) for i in live}
        got = d([(slabs[i], at[i], {k: v[at[i]:at[i] + n[i]] for k, v in x[i].items()}) for i in live], decode=decode)
        for i, o in zip(live, got):
            assert np.abs(o - want[i][at[i]:at[i] + n[i]]).max() <= tol, (i, at[i])
            at[i] += n[i]
        step += 1


@pytest.mark.parametrize("tokens,n_out,k", [(1, 128, 64), (1, 1000, 4096), (3, 300, 200), (16, 129, 72), (17, 512, 1000), (64, 4096, 2048),
                                             (255, 96, 328), (256, 640, 512), (300, 520, 136), (700, 1111, 1288), (33, 8, 8)])
@pytest.mark.parametrize("mode", ["bf16", "bf16->f32", "f32"])
def test_dense_gemm(tokens, n_out, k, mode):
    from lmdeploy_b200 import lib as l
    g = torch.Generator(device="cuda").manual_seed(tokens + n_out)
    td = torch.float32 if mode == "f32" else torch.bfloat16
    ldx, ldw, ldo = pad8(k) + 8, pad8(k), n_out + 3
    x = torch.full((tokens, ldx), float("nan"), dtype=td, device="cuda")
    w = torch.full((n_out, ldw), float("nan"), dtype=td, device="cuda")
    x[:, :k] = torch.randn(tokens, k, generator=g, device="cuda").to(td)
    w[:, :k] = torch.randn(n_out, k, generator=g, device="cuda").to(td)
    od = torch.bfloat16 if mode == "bf16" else torch.float32
    out = torch.full((tokens, ldo), 5.0, dtype=od, device="cuda")
    h = l.default_handle(0)
    for _ in range(2):                      # twice: split-k tickets reset themselves
        l.check(l.lib.tm_gemm_dense(h.ptr, out.data_ptr(), ldo, int(mode != "bf16"), x.data_ptr(), ldx, w.data_ptr(), ldw, tokens, n_out, k,
                                    int(mode == "f32"), torch.cuda.current_stream().cuda_stream), "tm_gemm_dense")
        h.check_device_status(torch.cuda.current_stream().cuda_stream)
    want = x[:, :k].double() @ w[:, :k].double().t()
    err = (out[:, :n_out].double() - want).abs().max().item() / k ** 0.5
    assert err <= (4e-2 if mode == "bf16" else 2e-5), err
    assert bool((out[:, n_out:] == 5.0).all())

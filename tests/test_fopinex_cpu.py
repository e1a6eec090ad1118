"""CPU: the plain restatement of the Fopinex mechanisms against other ways to say the same, and the parts of its serving path
that need no GPU."""
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import fopinex
from tests import fopinex_util as u

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_gated_linear_attention_is_decayed_linear_attention():
    rng = np.random.default_rng(1)
    n, d, e = 12, 5, 7
    q, k, v = (rng.standard_normal((n, 1, x)) for x in (d, d, e))
    a = rng.uniform(0.5, 1, (n, 1, d))
    o, s = fopinex.gated_linear_attention(q, k, v, a, np.zeros((1, d, e)))
    for t in range(n):
        want = sum((q[t, 0] * k[j, 0] * a[j + 1:t + 1, 0].prod(0)).sum() * v[j, 0] for j in range(t + 1))
        assert np.allclose(o[t, 0], want)
    o1, mid = fopinex.gated_linear_attention(q[:7], k[:7], v[:7], a[:7], np.zeros((1, d, e)))
    o2, end = fopinex.gated_linear_attention(q[7:], k[7:], v[7:], a[7:], mid)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(end, s)
    z = np.linspace(-30, 30, 61)
    assert np.allclose(np.log(fopinex.gla_decay(z, 4.0)) * 4, -np.logaddexp(0, -z))


@pytest.mark.parametrize("size", [0, 1, 4, 9, 100])
def test_chunks_are_counted_from_the_first_position(size):
    for i in range(60):
        first = fopinex.chunk_start(i, size)
        seen = [j for j in range(i + 1) if not size or j // size == i // size]
        assert seen == list(range(first, i + 1))


def test_mixed_attention_with_no_mixing_is_each_head_alone_and_mixing_is_linear():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 4, 6)), rng.standard_normal((9, 2, 6)), rng.standard_normal((9, 2, 5))
    bias, talk = rng.standard_normal(4), rng.standard_normal((4, 4))
    alone = fopinex.mixed_sigmoid_attention(q, k, v, 0.3, bias, np.eye(4))
    for h in range(4):
        w = np.tril(1 / (1 + np.exp(-(q[:, h] @ k[:, h // 2].T * 0.3 + bias[h]))))
        assert np.allclose(alone[:, h], w @ v[:, h // 2])
    # heads of one kv head share values, so mixing them is mixing their outputs
    one = v[:, :1]
    mixed = fopinex.mixed_sigmoid_attention(q, k[:, :1], one, 0.3, bias, talk, 4)
    single = fopinex.mixed_sigmoid_attention(q, k[:, :1], one, 0.3, bias, np.eye(4), 4)
    assert np.allclose(mixed, np.einsum("hg,tge->the", talk, single))
    # a portion at its place
    part = fopinex.mixed_sigmoid_attention(q[5:], k, v, 0.3, bias, talk, 4, first=5)
    assert np.allclose(part, fopinex.mixed_sigmoid_attention(q, k, v, 0.3, bias, talk, 4)[5:])


def test_routing():
    z = np.log(np.array([0.5, 0.3, 0.15, 0.05]))
    assert fopinex.route(z, np.zeros(4), 2)[0] == [0, 1]
    chosen, s = fopinex.route(z, np.array([0, -1.0, 0, 0.2]), 2)
    assert chosen == [0, 3] and np.allclose(s, [0.5, 0.05])            # weights without the correction, not renormalised
    # every choice score below zero: the experts of a group that is left out must not win as zeros
    chosen, _ = fopinex.route(z, np.array([-2.0, -0.6, -3.0, -3.0]), 2, 2, 1)
    assert chosen == [1, 0]
    assert fopinex.route(np.zeros(6), np.zeros(6), 3, 3, 2)[0] == [0, 1, 2]   # ties go to the lower index


def test_clamped_expert():
    h, one = np.array([1.0]), np.array([[1.0]])
    f = lambda g, u, limit: fopinex.clamped_expert(h, one * g, one * u, one, limit)[0]
    assert np.isclose(f(9.0, 0.0, 2.0), 2.0 / (1 + np.exp(-3.404)))             # the gate is cut above ...
    assert np.isclose(f(-9.0, 0.0, 2.0), -9.0 / (1 + np.exp(9 * 1.702)))        # ... and not below
    assert np.isclose(f(1.0, 5.0, 2.0), 3.0 * f(1.0, 0.0, 2.0)) and np.isclose(f(1.0, -5.0, 2.0), -f(1.0, 0.0, 2.0))


def test_architecture_is_known_and_its_command_lines_name_it():
    from lmdeploy_b200 import decoder
    assert "Fopinex" in decoder.architectures()
    r = subprocess.run([sys.executable, "-m", "lmdeploy_b200.generate", "--list"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0 and "Fopinex" in r.stdout


@pytest.mark.parametrize("cfg", [u.ODD, u.EVEN, u.ONES], ids=["odd", "even", "ones"])
def test_restatement_is_causal_and_layers_matter(cfg):
    w = u.weights(cfg, 3)
    ids = u.prompts(cfg, (24,))[0]
    a = u.oracle_logits(cfg, w, ids)
    assert np.isfinite(a).all() and np.allclose(a[:15], u.oracle_logits(cfg, w, ids[:15]))
    decay = f"l{[l['type'] for l in cfg['layers']].index('gla')}.mix.a2.b"
    for name in ("l0.mix.pb", "l0.mix.talk", decay, "l0.mlp.correction", "l0.rg1.b", "l0.rg2.b"):
        if name.endswith("correction") and cfg is not u.ODD:
            continue                                                           # nothing to choose
        changed = dict(w)
        changed[name] = w[name][::-1] * 1.5 + 0.25 * np.arange(w[name].size).reshape(w[name].shape)
        assert np.abs(u.oracle_logits(cfg, changed, ids) - a).max() > 1e-4, name

"""CPU: the plain restatement of the Rumazen mechanisms against other ways to say the same, and the parts of its serving
path that need no GPU (architecture table, slab manager, component library, replay command line)."""
import ctypes as C
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import rumazen
from tests import rumazen_util as u

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("size,pool", [(1, 1), (4, 3), (7, 2), (5, 8), (6, 0), (0, 0)])
def test_visible_keys_are_the_window_and_whole_blocks_behind_it(size, pool):
    for i in range(60):
        first, blocks = rumazen.visible(i, size, pool)
        tokens = [j for j in range(i + 1) if not size or i - j < size]
        assert tokens == list(range(first, i + 1))
        if size and pool:
            assert blocks == sum(1 for b in range(60) if b * pool + pool - 1 <= i - size)
            assert blocks * pool <= first                          # a block never overlaps the window
            assert first - blocks * pool < pool                    # less than a block is seen by nobody
        else:
            assert blocks == 0


def test_window_attention_with_everything_visible_is_plain_attention():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 4, 6)), rng.standard_normal((9, 2, 6)), rng.standard_normal((9, 2, 5))
    got = rumazen.window_attention(q, k, v, 0.3, softcap=2.0)
    for h in range(4):
        s = 2.0 * np.tanh(q[:, h] @ k[:, h // 2].T * 0.3 / 2.0)
        s[np.triu_indices(9, 1)] = -np.inf
        p = np.exp(s - s.max(1, keepdims=True))
        assert np.allclose(got[:, h], p / p.sum(1, keepdims=True) @ v[:, h // 2])


def test_delta_rule_is_a_product_of_transition_matrices():
    rng = np.random.default_rng(1)
    n, d = 12, 5
    r, k, v = (rng.standard_normal((n, 1, d)) for _ in range(3))
    w, a = rng.uniform(0.5, 1, (n, 1, d)), rng.uniform(0, 1, (n, 1, d))
    o, s = rumazen.delta_rule(r, k, v, w, a, np.zeros((1, d, d)))
    m = [np.diag(w[t, 0]) - np.outer(a[t, 0] * (uu := k[t, 0] / np.sqrt(k[t, 0] @ k[t, 0] + 1e-6)), uu) for t in range(n)]
    for t in range(n):
        total = np.zeros((d, d))
        for j in range(t + 1):
            x = np.outer(k[j, 0], v[j, 0])
            for i in range(j + 1, t + 1):
                x = m[i] @ x
            total += x
        assert np.allclose(o[t, 0], r[t, 0] @ total)
    assert np.allclose(s[0], total)
    # the same in two pieces
    o1, mid = rumazen.delta_rule(r[:7], k[:7], v[:7], w[:7], a[:7], np.zeros((1, d, d)))
    o2, end = rumazen.delta_rule(r[7:], k[7:], v[7:], w[7:], a[7:], mid)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(end, s)


def test_rotation_keeps_scores_a_function_of_the_distance():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    def score(i, j):
        return rumazen.rotate_interleaved(q, [i], 6, 50.0, 2.0)[0, 0] @ rumazen.rotate_interleaved(k, [j], 6, 50.0, 2.0)[0, 0]
    assert np.isclose(score(9, 4), score(25, 20)) and not np.isclose(score(9, 4), score(9, 5))
    same = rumazen.rotate_interleaved(q, [7], 6, 50.0)
    assert np.array_equal(same[..., 6:], q[..., 6:])
    assert np.isclose(same[0, 0, 0], q[0, 0, 0] * np.cos(7) - q[0, 0, 1] * np.sin(7))      # the first pair turns by the position


def test_gelu_and_norm():
    z = np.linspace(-6, 6, 101)
    assert np.allclose(rumazen.gelu_tanh(z), z * rumazen.sigmoid(2 * np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
    x = np.array([[3.0, 4.0]])
    assert np.allclose(rumazen.scalar_rms_norm(x, np.float32(2.0), 0.5), 2 * x / np.sqrt(12.5 + 0.5))


def test_architecture_table_names_both_models():
    from lmdeploy_b200 import decoder
    assert {"Rumazen", "turbomind-workspace"} <= set(decoder.architectures())


def test_slabs_of_a_model_s_own_layout_follow_the_manager_s_policy():
    from lmdeploy_b200 import lib as l
    m = C.c_void_p()
    assert l.lib.tm_cache_manager_create_slabs(C.byref(m), 1000, 64, 2, 1, -1) == l.TM_OK
    a, b, c = l.TmCacheSequence(), l.TmCacheSequence(), l.TmCacheSequence()
    assert l.lib.tm_cache_create(m, 1, None, C.byref(a)) == l.TM_OK
    assert l.lib.tm_cache_create(m, 2, None, C.byref(b)) == l.TM_OK
    assert abs(a.k_cache - b.k_cache) >= 1000
    assert l.lib.tm_cache_create(m, 3, None, C.byref(c)) == l.TM_ERR_WORKSPACE      # both slabs are in use
    assert l.lib.tm_cache_erase(m, 1) == l.TM_OK
    assert l.lib.tm_cache_create(m, 3, None, C.byref(c)) == l.TM_OK and c.k_cache == a.k_cache
    l.lib.tm_cache_manager_destroy(m)
    assert l.lib.tm_cache_manager_create_slabs(C.byref(m), 0, 64, 2, 1, -1) == l.TM_ERR_INVALID_ARG


def test_component_library_holds_the_decoder_and_no_more():
    from lmdeploy_b200 import build
    lib = C.CDLL(build.build(component="decoder"))
    for name in ("tm_create", "tm_model_open", "tm_model_prefill", "tm_model_decode", "tm_replay_step", "tm_cache_create"):
        assert hasattr(lib, name), name
    for name in ("tm_gemm_s4_f16", "tm_llama_create", "tm_sample_topk"):
        assert not hasattr(lib, name), name


def test_command_lines_explain_themselves():
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--help"], capture_output=True, text=True)
    assert r.returncode == 0 and "--max-tokens" in r.stdout
    r = subprocess.run([sys.executable, "-m", "lmdeploy_b200.generate", "--list"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 0 and "Rumazen" in r.stdout


def test_checkpoint_writer_round_trips(tmp_path):
    w = u.weights(u.ONES, 3)
    u.write_checkpoint(str(tmp_path), u.ONES, w)
    raw = open(tmp_path / "model.safetensors", "rb").read()
    import json
    n = int.from_bytes(raw[:8], "little")
    head = json.loads(raw[8:8 + n])
    s = head["l0.mix.q"]["data_offsets"]
    back = (np.frombuffer(raw[8 + n + s[0]:8 + n + s[1]], "<u2").astype(np.uint32) << 16).view(np.float32)
    assert np.array_equal(back.reshape(w["l0.mix.q"].shape), w["l0.mix.q"])

"""cpu: the plain restatement of the Gebadra design is consistent with itself (one call, token by token, portions), its
helpers do what their docstrings say, and the registry knows the family."""
import ctypes
import math
import os
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tests"))

import gebadra_oracle as O  # noqa: E402
import gebadra_util as U  # noqa: E402


def test_oracle_cut_invariance_and_shared_weights():
    layers = [U.lightning(mlp=U.dense()), U.parallel(mlp=U.dense(ff=5)), U.lightning(mlp=U.dense(), weights_of=0), U.parallel(mlp=None)]
    cfg = U.make_config(layers, width=12, vocab=19, streams=3)
    assert [O.weight_layer(cfg, i) for i in range(4)] == [0, 1, 0, 3]
    w = U.values(U.random_weights(cfg, seed=1))
    assert not any(n.startswith("l2.") for n in w) and "l3.norm2" not in w
    toks = [int(t) for t in np.random.default_rng(0).integers(0, 19, 21)]
    whole, stream = O.forward(cfg, w, toks)
    assert stream.shape == (4, 21, 12)
    st, rows, lay = O.Stepper(cfg, w), [], []
    for c0, c1 in ((0, 5), (5, 7), (7, 8), (8, 21)):
        lg, af = st.run(toks[c0:c1])
        rows.append(lg)
        lay.append(af)
    assert np.allclose(np.concatenate(rows), whole, rtol=1e-12, atol=1e-12)
    assert np.allclose(np.concatenate(lay, axis=1), stream, rtol=1e-12, atol=1e-12)


def test_layer_norm_and_streams():
    x = np.array([1.0, 3.0, 5.0, 7.0])
    out = O.layer_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), np.array([0.0, 0.0, 0.5, 0.0]), 0.0)
    s = math.sqrt(5.0)
    assert np.allclose(out, [-3 / s, -2 / s, 1 / s + 0.5, 3 / s])
    assert np.allclose(O.layer_norm(x, np.ones(4), np.zeros(4), 11.0), (x - 4.0) / 4.0)  # eps sits inside the root
    a, b = np.array([1.0, 0.0]), np.array([0.0, 1.0])
    assert np.allclose(O.streams_read([a, b], [2.0, 3.0]), [2.0, 3.0])
    new = O.streams_write([a, b], np.array([[1.0, 10.0], [100.0, 1000.0]]), [1.0, -1.0], np.array([0.5, 0.5]))
    assert np.allclose(new[0], [1.5, 100.5]) and np.allclose(new[1], [9.5, 999.5])  # mix[from, to], all from the old streams


def test_visible_tokens_and_blocks():
    # window 4, blocks of 3: block b is seen once its last token is four positions back or more
    assert O.visible(0, 4, 3) == ([], [0])
    assert O.visible(5, 4, 3) == ([], [2, 3, 4, 5])      # tokens 0 and 1 have left the window, block 0 is not yet seen
    assert O.visible(6, 4, 3) == ([0], [3, 4, 5, 6])
    assert O.visible(8, 4, 3) == ([0], [5, 6, 7, 8])
    assert O.visible(9, 4, 3) == ([0, 1], [6, 7, 8, 9])
    assert O.visible(7, 1, 1) == (list(range(7)), [7])   # blocks of one token: everything is seen
    assert O.visible(9, 2, 6) == ([0], [8, 9])


def test_rotation_pairs_and_scaling():
    rot = {"base": 100.0, "dims": 4}
    v = np.array([1.0, 2.0, 3.0, 4.0, 5.0])
    assert np.allclose(O.rotate_neighbours(v, 0, rot), v)
    out = O.rotate_neighbours(v, 3, rot)
    assert np.isclose(out[0], math.cos(3.0) - 2.0 * math.sin(3.0)) and np.isclose(out[1], 2.0 * math.cos(3.0) + math.sin(3.0))
    assert np.isclose(out[2], 3.0 * math.cos(0.3) - 4.0 * math.sin(0.3)) and out[4] == 5.0
    scaled = dict(rot, scaling={"factor": 4.0})
    assert np.allclose(O.rotate_neighbours(v, 12, scaled), O.rotate_neighbours(v, 3, rot))  # positions are divided by the factor
    q, k = np.arange(1.0, 5.0), np.array([0.5, -1.0, 2.0, 0.25])
    assert np.isclose(O.rotate_neighbours(q, 9, scaled) @ O.rotate_neighbours(k, 4, scaled), O.rotate_neighbours(q, 25, scaled) @ O.rotate_neighbours(k, 20, scaled))


def test_attention_pools_and_mixes_heads():
    # queries of zero: every visible key has the same weight, so the output is a mean of values that shows what took part
    mx = {"dim": 2, "heads": 2, "kv_heads": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 2, "pool": 2}}
    w = {"a.q": np.zeros((4, 1)), "a.k": np.zeros((2, 1)), "a.v": np.ones((1, 1)), "a.q.norm": np.ones(4), "a.k.norm": np.ones(2),
         "a.talk": np.array([[1.0, 0.0], [2.0, 1.0]]), "a.o": np.eye(2)}
    cache = []
    for t in range(5):
        y = O.talking_attention(w, "a.", mx, np.array([float(t)]), t, cache, 1e-6)
    # position 4 sees tokens 3 and 4 and the block of 0 and 1 (mean 0.5); block of 2 and 3 is not whole before the window
    assert np.isclose(y[0], (0.5 + 3.0 + 4.0) / 3.0) and np.isclose(y[1], 3.0 * y[0])


def test_linear_recurrence_decays_and_norms():
    st = np.zeros((1, 1, 1))
    outs = [float(O.decayed_outer_step(st, np.ones((1, 1)), np.ones((1, 1)), np.full((1, 1), v), [0.5])[0, 0]) for v in (4.0, 0.0, 1.0)]
    assert outs == [4.0, 2.0, 2.0]
    mx = {"heads": 1, "dim": 1, "vdim": 2, "decay": [0.9]}
    w = {"r.q": np.ones((1, 1)), "r.k": np.ones((1, 1)), "r.v": np.array([[3.0], [4.0]]), "r.g": np.full((2, 1), 50.0), "r.o": np.eye(2) / 50.0}
    y = O.retention_step(w, "r.", mx, np.ones(1), np.zeros((1, 1, 2)), 0.0)
    assert np.allclose(y, np.array([3.0, 4.0]) / math.sqrt(12.5))  # a unit norm per head, then the gate


def test_registry_knows_the_family():
    so = os.path.join(ROOT, "qwen_inference_engine_b200", "libqie_b200.so")
    if not os.path.exists(so):
        pytest.skip("library not built")
    lib = ctypes.CDLL(so)
    lib.qie_model_families.restype = ctypes.c_char_p
    assert "Gebadra" in lib.qie_model_families().decode().split(",")

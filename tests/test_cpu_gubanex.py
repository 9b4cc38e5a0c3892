"""cpu: the plain restatement of the Gubanex design is consistent with itself (one call, token by token, portions), its
helpers do what their docstrings say, the identities that the kernels use hold, and the registry knows the family."""
import ctypes
import math
import os
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tests"))

import gubanex_oracle as O  # noqa: E402
import gubanex_util as U  # noqa: E402


def test_oracle_cut_invariance_and_run_order():
    cfg = U.make_config([U.attention(mlp=U.moe()), U.gla(mlp=U.moe(top=1)), U.attention(size=0)], width=12, vocab=19, loop=(1, 2, 3))
    assert O.layer_runs(cfg) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]
    assert O.layer_runs(dict(cfg, loop={"start": 2, "stop": 2, "times": 4})) == [(0, None), (1, None), (2, None)]
    w = U.values(U.random_weights(cfg, seed=1))
    assert w["l1.mix.a1"].shape == (4, 12) and "l2.norm2" not in w
    toks = [int(t) for t in np.random.default_rng(0).integers(0, 19, 21)]
    whole, stream = O.forward(cfg, w, toks)
    assert stream.shape == (5, 21, 12)
    st, rows, lay = O.Stepper(cfg, w), [], []
    for c0, c1 in ((0, 5), (5, 7), (7, 8), (8, 21)):
        lg, af = st.run(toks[c0:c1])
        rows.append(lg)
        lay.append(af)
    assert np.allclose(np.concatenate(rows), whole, rtol=1e-12, atol=1e-12)
    assert np.allclose(np.concatenate(lay, axis=1), stream, rtol=1e-12, atol=1e-12)


def test_norms_cap_and_visibility():
    x = np.array([3.0, 4.0])
    assert np.allclose(O.unit_rms(x, 0.0), x / math.sqrt(12.5)) and np.allclose(O.unit_rms(x, 12.5), x / 5.0)  # eps sits inside the root
    assert np.allclose(O.zero_centred_norm(x, np.array([0.0, 1.0]), 12.5), [0.6, 1.6])
    assert np.isclose(O.softcap(1e9, 5.0), 5.0) and O.softcap(3.0, 0.0) == 3.0 and np.isclose(O.softcap(1.0, 2.0), 2.0 * math.tanh(0.5))
    assert O.visible(0, 4) == [0] and O.visible(3, 4) == [0, 1, 2, 3] and O.visible(4, 4) == [4] and O.visible(6, 4) == [4, 5, 6]
    assert O.visible(5, 1) == [5] and O.visible(2, 0) == [0, 1, 2]


def test_frequencies_by_wavelength():
    rot = {"base": 50.0, "dims": 8, "scaling": U.waves(3.0, 1.0, 4.0, 32)}
    f, plain = O.frequencies(rot), O.frequencies(rot, fault_unscaled=True)
    assert np.allclose(plain, [50.0 ** (-i / 4.0) for i in range(4)])
    assert f[0] == plain[0]                                  # wavelength 6.3 < 8: as it is
    assert np.isclose(f[2], plain[2] / 3.0) and np.isclose(f[3], plain[3] / 3.0)  # beyond 32: divided
    s = (32.0 / (2.0 * math.pi / plain[1]) - 1.0) / 3.0
    assert 0.0 < s < 1.0 and np.isclose(f[1], (1.0 - s) * plain[1] / 3.0 + s * plain[1])
    v = np.array([1.0, 2.0, 3.0, 4.0, 5.0])
    rot = {"base": 100.0, "dims": 4}
    out = O.rotate(v, 3, rot)
    assert np.isclose(out[0], math.cos(3.0) - 3.0 * math.sin(3.0)) and np.isclose(out[2], 3.0 * math.cos(3.0) + math.sin(3.0))
    assert np.isclose(out[1], 2.0 * math.cos(0.3) - 4.0 * math.sin(0.3)) and out[4] == 5.0
    # the rotation keeps the length, so a norm without a weight may stand before it or behind it
    assert np.allclose(O.unit_rms(out, 0.1), O.rotate(O.unit_rms(v, 0.1), 3, rot))


def test_attention_sees_its_chunk():
    # queries of zero: every visible key has the same weight, so the output is a mean of values that shows what took part
    mx = {"dim": 2, "heads": 2, "kv_heads": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 3}}
    w = {"a.q": np.zeros((4, 1)), "a.k": np.ones((2, 1)), "a.v": np.ones((1, 1)), "a.o": np.eye(2)}
    cache, out = [], []
    for t in range(5):
        out.append(O.chunked_attention(w, "a.", mx, np.array([float(t + 1)]), t, cache, 1e-6)[0])
    assert np.allclose(out, [1.0, 1.5, 2.0, 4.0, 4.5])


def test_gated_recurrence_and_its_chunked_form():
    mx = {"heads": 1, "dim": 2, "vdim": 1, "tau": 2.0}
    w = {"r.q": np.ones((2, 1)), "r.k": np.ones((2, 1)), "r.v": np.ones((1, 1)), "r.g": np.zeros((1, 1)), "r.o": np.eye(1), "r.norm": np.ones(1),
         "r.a1": np.zeros((1, 1)), "r.a2": np.zeros((2, 1)), "r.a2.b": np.array([0.0, 50.0])}
    assert np.allclose(O.channel_decay(w, "r.", mx, np.ones(1)), [[math.sqrt(0.5), 1.0]])
    st = np.zeros((1, 2, 1))
    for _ in range(3):
        O.gated_linear_step(w, "r.", mx, np.ones(1), st, 1e-6)
    r = math.sqrt(0.5)
    assert np.allclose(st[0, :, 0], [1.0 + r + 0.5, 3.0])
    # weights of pairs of tokens as products of decayed queries and keys around any reference of the running sums
    rng = np.random.default_rng(3)
    T, d, vd = 12, 5, 3
    q, k, v, g = rng.standard_normal((T, d)), rng.standard_normal((T, d)), rng.standard_normal((T, vd)), -rng.random((T, d))
    S, want = rng.standard_normal((d, vd)), []
    b, S0 = np.cumsum(g, axis=0), None
    S0 = S.copy()
    for t in range(T):
        S = np.exp(g[t])[:, None] * S + np.outer(k[t], v[t])
        want.append(S.T @ q[t])
    mid = 0.5 * (b[0] + b[-1])
    A = np.tril((q * np.exp(b - mid)) @ (k * np.exp(mid - b)).T)
    assert np.allclose((q * np.exp(b)) @ S0 + A @ v, want)
    assert np.allclose(np.exp(b[-1])[:, None] * S0 + (k * np.exp(b[-1] - b)).T @ v, S)


def test_router_and_scaled_inputs():
    chosen, weights = O.route(np.array([0.0, 3.0, -1.0, 3.0]), 3)
    assert chosen == [1, 3, 0] and np.allclose(weights, [O.sigmoid(3.0), O.sigmoid(3.0), 0.5])
    rng = np.random.default_rng(5)
    w = {"m.router": rng.standard_normal((3, 4)), **{f"m.e{e}.{n}": rng.standard_normal((6, 4) if n != "down" else (4, 6)) for e in range(3) for n in ("gate", "up", "down")}}
    h = rng.standard_normal(4)
    mlp = {"router": {"experts": 3, "top": 2}}
    got = O.expert_mixture(w, "m.", mlp, h)
    chosen, weights = O.route(w["m.router"] @ h, 2)
    want = np.zeros(4)
    for e, g in zip(chosen, weights):  # both linear maps let the factor through
        gate, up = g * (w[f"m.e{e}.gate"] @ h), g * (w[f"m.e{e}.up"] @ h)
        want += w[f"m.e{e}.down"] @ (O.silu(gate) * up)
    assert np.allclose(got, want)


def test_registry_knows_the_family():
    so = os.path.join(ROOT, "qwen_inference_engine_b200", "libqie_b200.so")
    if not os.path.exists(so):
        pytest.skip("library not built")
    lib = ctypes.CDLL(so)
    lib.qie_model_families.restype = ctypes.c_char_p
    assert "Gubanex" in lib.qie_model_families().decode().split(",")

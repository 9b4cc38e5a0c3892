"""gpu: the Gebadra family against the plain float64 restatement in tests/gebadra_oracle.py.

Every test builds its own small configuration and random bf16-exact weights, writes them as a model folder and loads
that through the model registry.  Most run in float32 so that a wrong key, window or block edge, rotation, head mix,
stream mix or lost state shows at 1e-4; where random weights would hide a fault the test first proves that the fault
WOULD show (the oracle with that mistake planted differs from the right answer by far more than the tolerance)."""
import copy
import os
import sys

import numpy as np
import pytest

torch = pytest.importorskip("torch")
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tests"))
pytestmark = pytest.mark.gpu

import gebadra_oracle as O  # noqa: E402
import gebadra_util as U  # noqa: E402

TOL32 = 2e-4


def _engine(tmp_path, cfg, weights, dtype="float32", page_size=16, max_pages=32, max_seqs=4, rows=256, name="m", use_graph=False):
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    import qwen_inference_engine_b200 as q
    folder = U.write_model(str(tmp_path / name), cfg, weights)
    return q.Engine(model_dir=folder, dtype=dtype, page_size=page_size, max_pages=max_pages, max_seqs=max_seqs,
                    max_batch_tokens=rows, context=page_size * max_pages, use_graph=use_graph)


def _tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def _runs(cfg, n, length, seed):
    """tokens in runs of `length` equal ones: the keys of a block point the same way, so its mean key keeps their size"""
    return [t for t in _tokens(cfg, (n + length - 1) // length, seed) for _ in range(length)][:n]


def _oracle_logits(cfg, weights, tokens, **kw):
    return O.forward(cfg, U.values(weights), tokens, **kw)[0]


def _whole(eng, tokens):
    s = eng.new_sequence()
    try:
        return eng.forward_batch([(s, tokens)], range(len(tokens)))
    finally:
        eng.free_sequence(s)


def _cuts(eng, tokens, cuts):
    assert sum(cuts) == len(tokens)
    s, at, rows = eng.new_sequence(), 0, []
    for c in cuts:
        rows.append(eng.forward_batch([(s, tokens[at:at + c])], range(c)))
        at += c
    eng.free_sequence(s)
    return np.concatenate(rows)


def _row_err(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1))


def _mixed_layers():
    return [U.parallel(mlp=U.dense()), U.lightning(mlp=U.dense(ff=9)), U.lightning(mlp=U.dense(ff=9), weights_of=1),
            U.parallel(heads=6, kv_heads=3, dim=4, vdim=5, size=5, pool=4, rot_dims=2, rheads=3, rdim=5, rvdim=3, mlp=None),
            U.parallel(mlp=U.dense(), weights_of=0)]


# ---------------------------------------------------------------------------------------------- each mechanism alone
SINGLE = {
    "lightning": ([U.lightning()], 2),
    "lightning_one_head": ([U.lightning(heads=1, dim=7, vdim=3, decay=[1.0])], 1),
    "lightning_wide_values": ([U.lightning(heads=2, dim=3, vdim=70, decay=[0.0, 0.9], mlp=U.dense(ff=3))], 3),
    "lightning_wide_keys": ([U.lightning(heads=2, dim=130, vdim=2)], 2),
    "lightning_long_row": ([U.lightning(heads=5, dim=4, vdim=103)], 2),
    "parallel": ([U.parallel()], 2),
    "parallel_plain": ([U.parallel(heads=3, kv_heads=3, dim=5, vdim=3, rot_dims=0, rheads=1)], 1),
    "parallel_one_kv_head": ([U.parallel(heads=8, kv_heads=1, dim=4, vdim=40, size=1, pool=1, rot_dims=4, factor=None)], 4),
    "parallel_one_head": ([U.parallel(heads=1, kv_heads=1, dim=7, vdim=2, size=4, pool=2, rot_dims=6, factor=3.0)], 5),
    "parallel_block_longer_than_window": ([U.parallel(size=3, pool=8)], 2),
    "parallel_block_longer_than_page": ([U.parallel(size=2, pool=20, rheads=3, rdim=9, rvdim=33)], 2),
    "parallel_many_value_columns": ([U.parallel(heads=12, kv_heads=12, dim=8, vdim=50, size=9, pool=5, rot_dims=8, mlp=U.dense())], 8),
    "shared_weights": ([U.parallel(mlp=U.dense()), U.parallel(mlp=U.dense(), weights_of=0), U.lightning(), U.lightning(weights_of=2)], 2),
    "shared_weights_in_a_row": ([U.lightning(mlp=U.dense()), U.lightning(mlp=U.dense(), weights_of=0), U.lightning(mlp=U.dense(), weights_of=1)], 3),
}


@pytest.mark.parametrize("name", list(SINGLE))
def test_single_mechanism_matches_oracle(tmp_path, name):
    layers, streams = SINGLE[name]
    cfg = U.make_config(copy.deepcopy(layers), width=20, vocab=37, streams=streams)
    w = U.random_weights(cfg, seed=3)
    toks = _tokens(cfg, 27, 1)
    eng = _engine(tmp_path, cfg, w)
    assert eng.family == "gebadra"
    eng.set_int("dump_layers", 1)
    got = _whole(eng, toks)
    want, stream_want = O.forward(cfg, U.values(w), toks)
    nr = len(layers)
    stream = eng.read_activation("layers", nr * 256 * cfg["width"], np.float32).reshape(nr, 256, cfg["width"])[:, :len(toks)]
    step = _cuts(eng, toks, [3, 2] + [1] * 22)
    eng.close()
    for i in range(nr):
        assert U.rel_err(stream[i], stream_want[i]) < TOL32, i
    assert U.rel_err(got, want) < TOL32
    assert U.rel_err(step, want) < TOL32


def test_other_sizes_and_constants(tmp_path):
    # other widths, eps, stream counts, a mixed order with and without feed-forwards (widths 30 and 17 are no multiples of 4:
    # the scalar paths of the norms and of the GEMV)
    for width, eps, streams in ((28, 1e-3, 3), (36, 1e-6, 1), (24, 1e-2, 6), (30, 1e-5, 2), (17, 1e-5, 7)):
        cfg = U.make_config(_mixed_layers(), width=width, vocab=41, eps=eps, streams=streams)
        w = U.random_weights(cfg, seed=11 + width)
        toks = _tokens(cfg, 30, 2)
        eng = _engine(tmp_path, cfg, w, name=f"m{width}")
        got = _whole(eng, toks)
        eng.close()
        assert U.rel_err(got, _oracle_logits(cfg, w, toks)) < TOL32


# ---------------------------------------------------------------------------------------------- cutting and batching
def test_prefill_decode_portions_and_batches_agree(tmp_path):
    cfg = U.make_config(_mixed_layers(), width=24, vocab=53, streams=3)
    w = U.random_weights(cfg, seed=5)
    reqs = [_tokens(cfg, n, 10 + i) for i, n in enumerate([41, 17, 2, 29])]
    want = [_oracle_logits(cfg, w, t) for t in reqs]
    eng = _engine(tmp_path, cfg, w, page_size=8, max_pages=24, rows=32)  # 41 tokens > 32 rows: the engine cuts, too
    for t, e in zip(reqs, want):
        assert U.rel_err(_whole(eng, t), e) < TOL32
    assert U.rel_err(_cuts(eng, reqs[0], [1] * 41), want[0]) < TOL32  # token by token
    for cuts in ([2, 2, 3, 9, 2, 16, 1, 1, 5], [7, 7, 7, 7, 7, 6], [40, 1], [1, 38, 2]):  # portions down to two tokens
        assert U.rel_err(_cuts(eng, reqs[0], cuts), want[0]) < TOL32
    # unequal requests together: portions of some beside single tokens of others
    seqs = [eng.new_sequence() for _ in reqs]
    at = [0] * len(reqs)
    got = [[] for _ in reqs]
    plan = [[5, 17, 1, 3], [1, 0, 1, 9], [20, 0, 0, 1], [1, 0, 0, 16], [14, 0, 0, 0]]
    for step in plan:
        entries, owner = [], []
        for i, c in enumerate(step):
            if c:
                entries.append((seqs[i], reqs[i][at[i]:at[i] + c]))
                owner += [i] * c
                at[i] += c
        lg = eng.forward_batch(entries, range(len(owner)))
        for row, i in zip(lg, owner):
            got[i].append(row)
    assert at == [len(t) for t in reqs]
    eng.close()
    for i in range(len(reqs)):
        assert U.rel_err(np.stack(got[i]), want[i]) < TOL32


def test_pages_and_slots_are_reused(tmp_path):
    # a pool of 8 pages of 8 positions and 2 slots: requests come and go; pages (with their pooled rows) and states get new owners
    cfg = U.make_config(_mixed_layers()[:3], width=20, vocab=31)
    w = U.random_weights(cfg, seed=7)
    eng = _engine(tmp_path, cfg, w, page_size=8, max_pages=8, max_seqs=2, rows=64)
    reqs = [_tokens(cfg, n, 30 + i) for i, n in enumerate([20, 27, 9, 24, 15, 30])]
    want = [_oracle_logits(cfg, w, t) for t in reqs]
    a = eng.new_sequence()
    b = eng.new_sequence()
    ga = [eng.forward_batch([(a, reqs[0][:11])], range(11))]
    gb = [eng.forward_batch([(b, reqs[1])], range(27))]
    ga.append(eng.forward_batch([(a, reqs[0][11:])], range(9)))
    assert U.rel_err(np.concatenate(ga), want[0]) < TOL32 and U.rel_err(gb[0], want[1]) < TOL32
    assert eng.pages_free() == 8 - 3 - 4
    with pytest.raises(Exception):
        eng.new_sequence()  # both slots live
    eng.free_sequence(a)
    for i in (2, 3):  # slot and pages of `a` serve two more requests while b stays: a stale state would move every token
        s = eng.new_sequence()
        lg = np.concatenate([eng.forward_batch([(s, reqs[i][:4])], range(4)), eng.forward_batch([(s, reqs[i][4:])], range(len(reqs[i]) - 4))])
        assert U.rel_err(lg, want[i]) < TOL32, i
        eng.free_sequence(s)
    eng.free_sequence(b)
    assert eng.pages_free() == 8
    s, t = eng.new_sequence(), eng.new_sequence()
    lg = eng.forward_batch([(s, reqs[4]), (t, reqs[5][:17])], range(15 + 17))
    lg2 = eng.forward_batch([(t, reqs[5][17:])], range(13))
    eng.close()
    assert U.rel_err(lg[:15], want[4]) < TOL32
    assert U.rel_err(np.concatenate([lg[15:], lg2]), want[5]) < TOL32


# ---------------------------------------------------------------------------------------------- edges that random weights hide
def _sharp(cfg, w, layer=0, factor=1.8, loud=2.0):
    """sharper scores and a louder left half: single keys carry the softmax and the mixer"""
    p = f"l{layer}.mix.left."
    for nm in ("q.norm", "k.norm"):
        U.set_values(w, p + nm, factor * w[p + nm][1])
    U.set_values(w, p + "out", loud * w[p + "out"][1])


def test_window_and_block_edges_in_prompts_and_decoding(tmp_path):
    # window 9 and blocks of 5 over pages of 4: no edge coincides with a page border for long, a block lies over two or three pages
    cfg = U.make_config([U.parallel(heads=4, kv_heads=2, dim=8, vdim=6, size=9, pool=5, scale=1.2, rot_dims=4, factor=2.0)], width=16, vocab=29)
    w = U.random_weights(cfg, seed=9, gain=2.0)
    _sharp(cfg, w)
    toks = _runs(cfg, 48, 5, 4)
    right = _oracle_logits(cfg, w, toks)
    for size, pool in ((10, 5), (8, 5), (9, 4), (9, 6)):  # the faults this test is about WOULD show
        bad = copy.deepcopy(cfg)
        bad["layers"][0]["mixer"]["left"]["mask"] = {"size": size, "pool": pool}
        assert U.rel_err(_oracle_logits(bad, w, toks)[16:], right[16:]) > 50 * TOL32, (size, pool)
    for kw in ({"fault_no_pool": True}, {"fault_pool_sees_early": 1}, {"fault_pool_sees_early": -1}):
        assert U.rel_err(_oracle_logits(cfg, w, toks, **kw)[14:], right[14:]) > 50 * TOL32, kw
    eng = _engine(tmp_path, cfg, w, page_size=4, max_pages=16, rows=64)
    assert U.rel_err(_whole(eng, toks), right) < TOL32                 # edges inside a prompt
    assert U.rel_err(_cuts(eng, toks, [5] + [1] * 43), right) < TOL32   # window and blocks pass over decoded tokens
    assert U.rel_err(_cuts(eng, toks, [2, 9, 3, 11, 2, 13, 8]), right) < TOL32  # blocks that several portions fill
    eng.close()


def test_far_block_among_hundreds_of_tokens(tmp_path):
    # 330 tokens behind a window of 20: about a hundred blocks of 3, several key tiles and pages, key splits when decoding
    cfg = U.make_config([U.parallel(heads=4, kv_heads=2, dim=8, vdim=6, size=20, pool=3, scale=1.3, rot_dims=6, base=1000.0)], width=16, vocab=23)
    w = U.random_weights(cfg, seed=13)
    _sharp(cfg, w, factor=2.2)
    toks = _tokens(cfg, 330, 6)
    right = _oracle_logits(cfg, w, toks)
    bad = toks[:3] + [(t + 1) % 23 for t in toks[3:6]] + toks[6:]  # another far block moves the last tokens
    assert U.rel_err(_oracle_logits(cfg, w, bad)[300:], right[300:]) > 5 * TOL32
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=24, rows=512)
    assert U.rel_err(_whole(eng, toks), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [285] + [1] * 45), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [100, 2, 61, 97, 70]), right) < TOL32
    eng.close()


def test_head_mix_norm_rotation_and_streams_are_what_decides(tmp_path):
    # each of these would go unnoticed with tame weights: the mix of the heads' weights, the norm over the whole projection,
    # the pairing and the scaling of the rotation, the orientation of the stream mix, a state of its own behind shared weights
    layers = [U.parallel(heads=4, kv_heads=2, dim=8, vdim=6, size=30, pool=4, scale=1.0, rot_dims=8, base=50.0, factor=3.0),
              U.lightning(heads=2, dim=6, vdim=5, mlp=U.dense()), U.lightning(heads=2, dim=6, vdim=5, mlp=U.dense(), weights_of=1)]
    cfg = U.make_config(layers, width=16, vocab=23, streams=3)
    w = U.random_weights(cfg, seed=23)
    _sharp(cfg, w)
    toks = _tokens(cfg, 90, 3)
    right = _oracle_logits(cfg, w, toks)
    for kw in ({"pairing": "half"}, {"fault_unscaled": True}, {"fault_no_talk": True}, {"fault_per_head_norm": True}, {"fault_transposed": True},
               {"fault_shared_state": True}):
        assert U.rel_err(_oracle_logits(cfg, w, toks, **kw)[20:], right[20:]) > 50 * TOL32, kw
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=8, rows=128)
    assert U.rel_err(_whole(eng, toks), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [70] + [1] * 20), right) < TOL32
    eng.close()


def test_states_survive_cuts_batches_and_long_portions(tmp_path):
    # slow decays: a state lost or mixed up at a cut moves everything after it
    slow = [0.999, 0.98]
    cfg = U.make_config([U.lightning(heads=2, dim=12, vdim=40, decay=slow, mlp=U.dense(ff=8)), U.parallel(rheads=2, rdim=7, rvdim=9, decay=slow)],
                        width=16, vocab=29)
    w = U.random_weights(cfg, seed=29)
    a, b = _tokens(cfg, 240, 7), _tokens(cfg, 110, 8)
    ra, rb = _oracle_logits(cfg, w, a), _oracle_logits(cfg, w, b)
    st = O.Stepper(cfg, U.values(w))  # the fault WOULD show: the second portion from a zero state
    assert U.rel_err(st.run(a[200:])[0], ra[200:]) > 50 * TOL32
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=40, rows=512)
    sa, sb = eng.new_sequence(), eng.new_sequence()
    lg = eng.forward_batch([(sa, a[:200]), (sb, b[:90])], range(290))
    assert U.rel_err(lg[:200], ra[:200]) < TOL32 and U.rel_err(lg[200:], rb[:90]) < TOL32
    lg = eng.forward_batch([(sb, b[90:]), (sa, a[200:202])], range(22))  # the carried states go on, in another order
    assert U.rel_err(lg[:20], rb[90:]) < TOL32 and U.rel_err(lg[20:], ra[200:202]) < TOL32
    tail = np.concatenate([eng.forward_batch([(sa, [t])], [0]) for t in a[202:]])
    assert U.rel_err(tail, ra[202:]) < TOL32
    eng.close()


def test_first_tokens_and_long_decoding(tmp_path):
    # the first tokens (a single key, a zero state) and 200 decoded tokens with windows and blocks passing over them
    cfg = U.make_config(_mixed_layers(), width=20, vocab=31)
    w = U.random_weights(cfg, seed=17)
    toks = _tokens(cfg, 203, 8)
    right = _oracle_logits(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=16, rows=64)
    got = _cuts(eng, toks, [1] * 203)
    eng.close()
    assert U.rel_err(got[:4], right[:4]) < TOL32
    assert U.rel_err(got, right) < TOL32


# ---------------------------------------------------------------------------------------------- generation and serving precision
def test_greedy_generation_through_engine_and_scheduler(tmp_path):
    import qwen_inference_engine_b200 as q
    cfg = U.make_config(_mixed_layers()[:4], width=24, vocab=61)
    w = U.random_weights(cfg, seed=21, gain=1.5)
    vals = U.values(w)
    prompts = [_tokens(cfg, n, 40 + i) for i, n in enumerate([9, 14, 5])]

    def greedy(prompt, n_new):
        st, out = O.Stepper(cfg, vals), []
        z = st.run(prompt)[0][-1]
        for _ in range(n_new):
            srt = np.sort(z)
            if srt[-1] - srt[-2] < 1e-3:  # a close call is not a fault of either side
                break
            out.append(int(np.argmax(z)))
            z = st.run([out[-1]])[0][-1]
        return out

    want = [greedy(p, 12) for p in prompts]
    assert sum(len(e) for e in want) > 20
    for use_graph in (False, True):  # eager launches, then decode steps replayed from CUDA graphs
        eng = _engine(tmp_path, cfg, w, page_size=8, max_pages=12, max_seqs=2, rows=64, name=f"g{int(use_graph)}", use_graph=use_graph)
        for p, e in zip(prompts, want):  # the engine's own entry point: prefill + decode steps
            assert eng.generate(p, 12)[:len(e)] == e
        free0 = eng.pages_free()
        sch = q.Scheduler(eng, max_running=2, eos_token=-1)  # three requests over two slots: the third waits for a slot
        rids = [sch.submit(p, 12) for p in prompts]
        sch.run()
        for rid, e in zip(rids, want):
            toks, fin = sch.result(rid)
            assert fin and toks[:len(e)] == e
        sch.close()
        assert eng.pages_free() == free0
        eng.close()


def test_top_k_sampling_draws_from_the_best_tokens(tmp_path):
    # with top-k 3 every drawn token is among the three largest logits of its position (the oracle's, where the third and fourth
    # are clearly apart), and top-k 1 is the greedy choice
    cfg = U.make_config(_mixed_layers()[:3], width=24, vocab=61)
    w = U.random_weights(cfg, seed=41, gain=1.5)
    prompt = _tokens(cfg, 11, 3)
    eng = _engine(tmp_path, cfg, w, page_size=8, max_pages=12, max_seqs=2, rows=64)
    greedy = eng.generate(prompt, 6)
    eng.set_sampling(topk=1)
    assert eng.generate(prompt, 6) == greedy
    eng.set_sampling(topk=3, temperature_prefill=1.0, temperature_decode=1.0, seed=7)
    drawn = eng.generate(prompt, 8)
    eng.close()
    st = O.Stepper(cfg, U.values(w))
    z = st.run(prompt)[0][-1]
    for t in drawn:
        order = np.argsort(z)[::-1]
        if z[order[2]] - z[order[3]] > 1e-3:
            assert t in order[:3]
        z = st.run([t])[0][-1]


def _tc_layers():
    # shapes the tensor-core kernels take: width 64, projections of 128 columns and more, head sizes that need padding
    return [U.parallel(heads=4, kv_heads=2, dim=24, vdim=20, size=37, pool=6, scale=0.5, rot_dims=8, rheads=2, rdim=20, rvdim=32, decay=[0.9, 0.998],
                       mlp=U.dense(ff=64)),
            U.lightning(heads=2, dim=24, vdim=32, decay=[0.7, 0.995], mlp=U.dense(ff=128)),
            U.lightning(heads=2, dim=24, vdim=32, decay=[0.7, 0.995], mlp=U.dense(ff=128), weights_of=1),
            U.parallel(heads=4, kv_heads=4, dim=40, vdim=48, size=100, pool=16, scale=0.3, rot_dims=40, factor=4.0, rheads=4, rdim=72, rvdim=16,
                       decay=[0.5, 0.9, 0.99, 1.0], mlp=None)]


def test_bf16_tensor_core_paths_keep_the_edges(tmp_path):
    # bf16 serving precision: tcgen05 GEMMs between bf16 rows, tensor-core attention with pooled rows (more than one block of 64 of
    # them) and two sequences of unequal length, chunks of the linear recurrence cut at segment ends and carried into the next call
    cfg = U.make_config(_tc_layers(), width=64, vocab=29, streams=2)
    w = U.random_weights(cfg, seed=31, gain=1.5)
    _sharp(cfg, w, 0, factor=1.4, loud=6.0)
    reqs = [_runs(cfg, 460, 3, 4), _runs(cfg, 81, 3, 5)]
    right = [_oracle_logits(cfg, w, t) for t in reqs]
    tol = 3e-2
    for size, pool in ((38, 6), (36, 6), (37, 5)):  # with a window or a block one key off a tenth of the rows is far over the tolerance
        bad = copy.deepcopy(cfg)
        bad["layers"][0]["mixer"]["left"]["mask"] = {"size": size, "pool": pool}
        assert np.quantile(_row_err(_oracle_logits(bad, w, reqs[0][:160]), right[0][:160])[44:], 0.9) > 2 * tol, (size, pool)
    assert np.median(_row_err(_oracle_logits(cfg, w, reqs[0][:160], fault_no_talk=True), right[0][:160])) > 2 * tol
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=72, rows=512)
    a, b = eng.new_sequence(), eng.new_sequence()
    lg = eng.forward_batch([(a, reqs[0][:400]), (b, reqs[1][:70])], range(470))
    lg2 = eng.forward_batch([(b, reqs[1][70:]), (a, reqs[0][400:403])], range(14))  # the per-row kernels over the same bf16 rows
    lg3 = eng.forward_batch([(a, reqs[0][403:])], range(57))
    whole = _whole(eng, reqs[0])
    eng.close()
    ea = _row_err(np.concatenate([lg[:400], lg2[11:], lg3]), right[0])
    eb = _row_err(np.concatenate([lg[400:], lg2[:11]]), right[1])
    ew = _row_err(whole, right[0])
    for err in (ea, eb, ew):
        assert np.median(err) < tol / 2 and np.quantile(err, 0.9) < tol, (np.median(err), err.max())


def test_bf16_other_sizes(tmp_path):
    # bf16 serving precision away from the tensor-core shapes: a width that is no multiple of 64, head sizes beyond the
    # tensor-core kernels' tiles, more value columns than one CTA of either attention kernel takes, portions against the whole
    layers = [U.parallel(heads=8, kv_heads=8, dim=40, vdim=72, size=50, pool=7, scale=0.3, rot_dims=10, rheads=2, rdim=136, rvdim=12, mlp=U.dense(ff=30)),
              U.lightning(heads=3, dim=9, vdim=130, mlp=None)]
    cfg = U.make_config(layers, width=36, vocab=41)
    w = U.random_weights(cfg, seed=37)
    toks = _tokens(cfg, 120, 9)
    right = _oracle_logits(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=24, rows=256)
    whole = _whole(eng, toks)
    cut = _cuts(eng, toks, [70, 3, 1, 46])
    eng.close()
    for got in (whole, cut):
        err = _row_err(got, right)
        assert np.median(err) < 1e-2 and np.quantile(err, 0.95) < 3e-2, (np.median(err), err.max())


@pytest.mark.parametrize("dim,vdim", [(16, 16), (64, 64), (80, 64), (64, 128), (128, 96), (20, 12)])
def test_bf16_linear_recurrence_in_chunks(tmp_path, dim, vdim):
    # the chunked form at every tile size, with decays from almost none to total, against the token-by-token form of a copy that
    # is fed in short portions: three sequences in a batch, portions that end inside, at and just behind a chunk of 64
    cfg = U.make_config([U.lightning(heads=4, dim=dim, vdim=vdim, decay=[0.0, 0.6, 0.99, 1.0])], width=64, vocab=29)
    w = U.random_weights(cfg, seed=43)
    reqs = [_tokens(cfg, n, 50 + i) for i, n in enumerate([193, 64, 130])]
    right = [_oracle_logits(cfg, w, t) for t in reqs]
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=40, rows=256)
    seqs = [eng.new_sequence() for _ in reqs]
    lg = eng.forward_batch([(seqs[0], reqs[0][:65]), (seqs[1], reqs[1]), (seqs[2], reqs[2][:1])], range(130))
    lg2 = eng.forward_batch([(seqs[2], reqs[2][1:]), (seqs[0], reqs[0][65:192])], range(256))
    lg3 = eng.forward_batch([(seqs[0], reqs[0][192:])], [0])
    steps = _cuts(eng, reqs[2], [2] * 65)
    eng.close()
    got = [np.concatenate([lg[:65], lg2[129:], lg3]), lg[65:129], np.concatenate([lg[129:], lg2[:129]])]
    for g, r in zip(got, right):
        err = _row_err(g, r)
        assert np.median(err) < 1e-2 and err.max() < 4e-2, (np.median(err), err.max())
    err = _row_err(steps, right[2])
    assert np.median(err) < 1e-2 and err.max() < 4e-2


@pytest.mark.parametrize("kv_heads,dim,vdim,size,pool,page", [
    (2, 64, 64, 100, 16, 64),    # a tile of keys is one page
    (2, 16, 32, 90, 16, 128),    # a page is two tiles
    (4, 40, 72, 70, 7, 16),      # 288 value columns: two chunks; blocks over page borders
    (2, 128, 128, 130, 32, 16),  # two blocks of head columns, fewer stages
    (1, 72, 24, 40, 16, 12),     # pages that do not divide a tile: every row by its own address
    (2, 32, 16, 9, 1, 16),       # blocks of one token: more tiles of pooled rows than stages
    (4, 8, 8, 500, 5, 32),       # a window longer than the prompt
], ids=["page64", "page128", "two_value_chunks", "wide_heads", "odd_pages", "blocks_of_one", "no_block_seen"])
def test_bf16_prompt_attention_tiles(tmp_path, kv_heads, dim, vdim, size, pool, page):
    # the tensor-core prompt attention (portions of 128 rows and more) against the restatement, and against short portions of the
    # same prompt through the other kernels; runs of equal tokens keep the pooled keys large, and the left half is loud
    cfg = U.make_config([U.parallel(heads=8, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size, pool=pool, scale=0.7 / np.sqrt(dim) * 2, rot_dims=dim // 4 * 2,
                                    factor=2.0, rheads=2, rdim=8, rvdim=8)], width=64, vocab=29)
    w = U.random_weights(cfg, seed=47, gain=1.3)
    _sharp(cfg, w, factor=1.2, loud=3.0)
    toks = _runs(cfg, 300, 3, 9)
    right = _oracle_logits(cfg, w, toks)
    other = _runs(cfg, 140, 3, 10)
    right2 = _oracle_logits(cfg, w, other)
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=page, max_pages=1600 // page, rows=512)
    whole = _whole(eng, toks)
    a, b = eng.new_sequence(), eng.new_sequence()
    first = eng.forward_batch([(a, toks[:131])], range(131))
    both = eng.forward_batch([(b, other), (a, toks[131:])], range(309))  # two sequences, one continues its cache
    eng.free_sequence(a)
    cut = _cuts(eng, toks, [60, 2, 63, 50, 1, 61, 63])
    eng.close()
    for got, want in ((whole, right), (np.concatenate([first, both[140:]]), right), (both[:140], right2), (cut, right)):
        err = _row_err(got, want)
        assert np.median(err) < 1e-2 and np.quantile(err, 0.95) < 3e-2 and err.max() < 8e-2, (np.median(err), err.max())
    assert np.median(_row_err(_oracle_logits(cfg, w, toks[:150], fault_no_talk=True), right[:150])) > 0.1

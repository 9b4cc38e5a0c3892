"""gpu: the Gubanex family against the plain float64 restatement in tests/gubanex_oracle.py.

Every test builds its own small configuration and random bf16-exact weights, writes them as a model folder and loads
that through the model registry.  Most run in float32 so that a wrong key, chunk edge, rotation, decay, expert weight or
lost state shows at 1e-4; where random weights would hide a fault the test first proves that the fault WOULD show (the
oracle with that mistake planted differs from the right answer by far more than the tolerance)."""
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

import gubanex_oracle as O  # noqa: E402
import gubanex_util as U  # noqa: E402

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
    return [U.attention(mlp=U.moe()), U.gla(mlp=U.moe(experts=4, top=1, ff=9)), U.attention(heads=6, kv_heads=3, dim=4, vdim=7, size=5, rot_dims=2, mlp=None),
            U.gla(heads=2, dim=5, vdim=9, tau=2.0, mlp=U.moe(experts=3, top=3, ff=5))]


# ---------------------------------------------------------------------------------------------- each mechanism alone
SINGLE = {
    "attention": ([U.attention()], None),
    "attention_no_sharing": ([U.attention(heads=3, kv_heads=3, dim=5, vdim=8, rot_dims=4)], None),
    "attention_one_kv_head": ([U.attention(heads=8, kv_heads=1, dim=4, vdim=40, size=3, rot_dims=4)], None),
    "attention_one_head": ([U.attention(heads=1, kv_heads=1, dim=7, vdim=2, size=4, rot_dims=6)], None),
    "attention_chunks_of_one": ([U.attention(size=1)], None),
    "attention_no_chunks": ([U.attention(size=0)], None),
    "attention_no_rotation": ([U.attention(rot_dims=0)], None),
    "attention_plain_frequencies": ([U.attention(dim=8, rot_dims=8, scaling={})], None),
    "attention_scaled_frequencies": ([U.attention(dim=10, rot_dims=10, base=30.0, scaling=U.waves(5.0, 0.5, 3.0, 20))], None),
    "gla": ([U.gla()], None),
    "gla_one_head": ([U.gla(heads=1, dim=7, vdim=3, tau=1.0)], None),
    "gla_wide_values": ([U.gla(heads=2, dim=3, vdim=70, tau=16.0)], None),
    "gla_wide_keys": ([U.gla(heads=2, dim=130, vdim=2)], None),
    "experts_one_chosen": ([U.gla(mlp=U.moe(experts=6, top=1))], None),
    "experts_all_chosen": ([U.gla(mlp=U.moe(experts=4, top=4, ff=3))], None),
    "one_expert": ([U.attention(mlp=U.moe(experts=1, top=1, ff=11))], None),
    "many_experts": ([U.attention(mlp=U.moe(experts=40, top=5, ff=4))], None),
    "loop_inside": ([U.attention(), U.gla(mlp=U.moe()), U.attention(mlp=U.moe()), U.gla()], (1, 3, 3)),
    "loop_whole_model": ([U.gla(), U.attention(mlp=U.moe())], (0, 2, 2)),
    "loop_at_the_end": ([U.gla(), U.attention(mlp=U.moe())], (1, 2, 4)),
    "loop_one_pass": ([U.gla(), U.attention()], (0, 1, 1)),
    "loop_empty": ([U.gla(), U.attention()], (1, 1, 5)),
}


@pytest.mark.parametrize("name", list(SINGLE))
def test_single_mechanism_matches_oracle(tmp_path, name):
    layers, loop = SINGLE[name]
    cfg = U.make_config(copy.deepcopy(layers), width=20, vocab=37, loop=loop)
    w = U.random_weights(cfg, seed=3)
    toks = _tokens(cfg, 27, 1)
    eng = _engine(tmp_path, cfg, w)
    assert eng.family == "gubanex"
    eng.set_int("dump_layers", 1)
    got = _whole(eng, toks)
    want, stream_want = O.forward(cfg, U.values(w), toks)
    nr = len(O.layer_runs(cfg))
    stream = eng.read_activation("layers", nr * 256 * cfg["width"], np.float32).reshape(nr, 256, cfg["width"])[:, :len(toks)]
    step = _cuts(eng, toks, [3, 2] + [1] * 22)
    eng.close()
    for i in range(nr):
        assert U.rel_err(stream[i], stream_want[i]) < TOL32, i
    assert U.rel_err(got, want) < TOL32
    assert U.rel_err(step, want) < TOL32


def test_other_sizes_and_constants(tmp_path):
    # other widths, eps, scales, caps and ranks (widths 30 and 17 are no multiples of 4: the scalar paths of the norms and of the GEMV;
    # width 1060 takes two pieces of the stream per thread)
    for width, eps, es, ls, cap, rank in ((28, 1e-3, 0.5, 2.0, 3.0, 1), (36, 1e-6, 7.0, 1.0, 0.0, 20), (24, 1e-2, 1.0, 0.3, 50.0, 33),
                                          (30, 1e-5, 3.0, 1.0, 5.0, 2), (17, 1e-5, 1.5, 0.7, 0.0, 3), (1060, 1e-5, 2.0, 0.4, 9.0, 4)):
        cfg = U.make_config(_mixed_layers(), width=width, vocab=41, eps=eps, embed_scale=es, logit_scale=ls, softcap=cap, loop=(1, 3, 2))
        w = U.random_weights(cfg, seed=11 + width, rank=rank)
        toks = _tokens(cfg, 30, 2)
        eng = _engine(tmp_path, cfg, w, name=f"m{width}")
        got = _whole(eng, toks)
        eng.close()
        assert U.rel_err(got, _oracle_logits(cfg, w, toks)) < TOL32, width


# ---------------------------------------------------------------------------------------------- cutting and batching
def test_prefill_decode_portions_and_batches_agree(tmp_path):
    cfg = U.make_config(_mixed_layers(), width=24, vocab=53, loop=(0, 2, 2))
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
    # a pool of 8 pages of 8 positions and 2 slots: requests come and go; pages and states get new owners
    cfg = U.make_config(_mixed_layers()[:2], width=20, vocab=31, loop=(0, 2, 2))
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
def test_chunk_edges_in_prompts_and_decoding(tmp_path):
    # chunks of 9 over pages of 4: no edge coincides with a page border for long; sharp scores, so single keys carry the softmax
    cfg = U.make_config([U.attention(heads=4, kv_heads=2, dim=8, vdim=6, size=9, scale=1.1, rot_dims=4)], width=16, vocab=29)
    w = U.random_weights(cfg, seed=9, gain=2.0)
    toks = _tokens(cfg, 48, 4)
    right = _oracle_logits(cfg, w, toks)
    for kw in ({"fault_chunk_shift": 1}, {"fault_chunk_shift": 8}, {"fault_window": True}):  # the faults this test is about WOULD show
        assert U.rel_err(_oracle_logits(cfg, w, toks, mixer=kw)[9:], right[9:]) > 50 * TOL32, kw
    for size in (8, 10):
        bad = copy.deepcopy(cfg)
        bad["layers"][0]["mixer"]["mask"]["size"] = size
        assert U.rel_err(_oracle_logits(bad, w, toks)[9:], right[9:]) > 50 * TOL32, size
    eng = _engine(tmp_path, cfg, w, page_size=4, max_pages=16, rows=64)
    assert U.rel_err(_whole(eng, toks), right) < TOL32                 # edges inside a prompt
    assert U.rel_err(_cuts(eng, toks, [5] + [1] * 43), right) < TOL32   # chunks begin and end on decoded tokens
    for cuts in ([2, 9, 3, 11, 2, 13, 8], [9, 9, 9, 9, 9, 3], [8, 2, 8, 10, 20]):  # portions that end on, before and behind an edge
        assert U.rel_err(_cuts(eng, toks, cuts), right) < TOL32, cuts
    eng.close()


def test_far_key_among_hundreds(tmp_path):
    # one key stands out: in its chunk of 300 tokens the token 7 occurs once, near the start, and queries find it; several key tiles,
    # pages and key splits lie between
    cfg = U.make_config([U.attention(heads=4, kv_heads=2, dim=8, vdim=6, size=300, scale=1.6, rot_dims=2, base=1e6, scaling={})], width=16, vocab=23)
    w = U.random_weights(cfg, seed=13, gain=1.5)
    toks = [t if t != 7 else 8 for t in _tokens(cfg, 380, 6)]
    toks[11] = 7
    toks[303] = 7  # the second chunk has one of its own
    right = _oracle_logits(cfg, w, toks)
    bad = list(toks)
    bad[11] = 5
    assert U.rel_err(_oracle_logits(cfg, w, bad)[250:300], right[250:300]) > 20 * TOL32
    assert U.rel_err(_oracle_logits(cfg, w, bad)[300:], right[300:]) < 1e-12  # beyond the chunk it is not seen
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=24, rows=512)
    assert U.rel_err(_whole(eng, toks), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [255] + [1] * 125), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [100, 2, 61, 97, 120]), right) < TOL32
    eng.close()


def test_what_tame_weights_hide(tmp_path):
    # each of these would go unnoticed with tame weights: pairing and scaling of the rotation, the norm behind it, the order of the head
    # groups, tau, a decay per channel, what the decay acts on, the query scale, where the router's weight enters, a state of its own
    # per pass, the embedding before a pass, zero-centred weights, the logits' scale and cap
    layers = [U.attention(heads=4, kv_heads=2, dim=8, vdim=6, size=30, scale=1.0, rot_dims=8, base=50.0, mlp=U.moe(experts=4, top=2)),
              U.gla(heads=2, dim=6, vdim=5, tau=3.0, mlp=U.moe(experts=5, top=1))]
    cfg = U.make_config(layers, width=16, vocab=23, loop=(0, 2, 2))
    w = U.random_weights(cfg, seed=23, gain=1.5)
    for i in (1,):  # decays between fast and slow, different from channel to channel
        U.set_values(w, f"l{i}.mix.a2.b", np.linspace(-3.0, 6.0, 12))
    toks = _tokens(cfg, 90, 3)
    right = _oracle_logits(cfg, w, toks)
    for kw in ({"mixer": {"pairing": "neighbours"}}, {"mixer": {"fault_unscaled": True}}, {"mixer": {"fault_no_blend": True}},
               {"mixer": {"fault_no_qk_norm": True}}, {"mixer": {"fault_heads_interleaved": True}}, {"linear": {"fault_no_tau": True}},
               {"linear": {"fault_head_decay": True}}, {"linear": {"fault_decay_after": True}}, {"linear": {"fault_no_q_scale": True}},
               {"mlp": {"fault_output_weight": True}}, {"mlp": {"fault_renormalised": True}}, {"fault_shared_passes": True},
               {"fault_no_reentry": True}, {"fault_plain_weight": True}):
        # (the norm per head takes a scale of the queries out again, but for its eps)
        bound = 50 * TOL32 if kw != {"linear": {"fault_no_q_scale": True}} else 0.0
        assert U.rel_err(_oracle_logits(cfg, w, toks, **kw)[20:], right[20:]) > bound, kw
    for key, val in (("logit_softcap", 0.0), ("logit_scale", 1.0)):
        assert U.rel_err(_oracle_logits(dict(cfg, **{key: val}), w, toks), right) > 50 * TOL32, key
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=8, rows=128)
    assert U.rel_err(_whole(eng, toks), right) < TOL32
    assert U.rel_err(_cuts(eng, toks, [70] + [1] * 20), right) < TOL32
    eng.close()


def test_query_scale_shows_when_eps_is_large(tmp_path):
    # the norm behind the recurrence hides a scale of the queries unless eps is comparable to their products
    cfg = U.make_config([U.gla(heads=2, dim=9, vdim=4)], width=16, vocab=23, eps=0.5)
    w = U.random_weights(cfg, seed=25)
    toks = _tokens(cfg, 20, 3)
    right = _oracle_logits(cfg, w, toks)
    assert U.rel_err(_oracle_logits(cfg, w, toks, linear={"fault_no_q_scale": True}), right) > 50 * TOL32
    eng = _engine(tmp_path, cfg, w)
    assert U.rel_err(_whole(eng, toks), right) < TOL32
    eng.close()


def test_states_survive_cuts_batches_and_long_portions(tmp_path):
    # slow decays: a state lost or mixed up at a cut moves everything after it
    cfg = U.make_config([U.gla(heads=2, dim=12, vdim=40, tau=16.0, mlp=U.moe(experts=2, top=1, ff=8)), U.gla(heads=2, dim=7, vdim=9, tau=8.0)], width=16, vocab=29)
    w = U.random_weights(cfg, seed=29)
    for i in (0, 1):
        b = w[f"l{i}.mix.a2.b"][1]
        U.set_values(w, f"l{i}.mix.a2.b", 3.0 + np.abs(b))
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
    # the first tokens (a single key, a zero state) and 200 decoded tokens with chunks passing over them
    cfg = U.make_config(_mixed_layers(), width=20, vocab=31, loop=(1, 4, 2))
    w = U.random_weights(cfg, seed=17)
    toks = _tokens(cfg, 203, 8)
    right = _oracle_logits(cfg, w, toks)
    eng = _engine(tmp_path, cfg, w, page_size=16, max_pages=16, rows=64)
    got = _cuts(eng, toks, [1] * 203)
    eng.close()
    assert U.rel_err(got[:4], right[:4]) < TOL32
    assert U.rel_err(got, right) < TOL32


# ---------------------------------------------------------------------------------------------- generation
def test_greedy_generation_through_engine_and_scheduler(tmp_path):
    import qwen_inference_engine_b200 as q
    cfg = U.make_config(_mixed_layers(), width=24, vocab=61, loop=(0, 2, 2))
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
    cfg = U.make_config(_mixed_layers()[:3], width=24, vocab=61, softcap=30.0)
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
        if z[order[2]] - z[order[3]] > 0.05:  # (the sampler reads bf16 logits)
            assert t in order[:3]
        z = st.run([t])[0][-1]


# ---------------------------------------------------------------------------------------------- serving precision
def test_bf16_tensor_core_paths_keep_the_edges(tmp_path):
    # bf16 serving precision: tcgen05 GEMMs between bf16 rows, the store from bf16 rows, tensor-core attention with a chunk's edge inside
    # a tile, the chunked recurrence carried over calls, grouped expert GEMMs (every expert chosen: no close calls); two sequences of
    # unequal length
    layers = [U.attention(heads=4, kv_heads=2, dim=32, vdim=24, size=37, scale=0.25, rot_dims=16, mlp=U.moe(experts=3, top=3, ff=64)),
              U.gla(heads=2, dim=24, vdim=32, tau=8.0, mlp=U.moe(experts=2, top=2, ff=32)),
              U.attention(heads=2, kv_heads=2, dim=48, vdim=64, size=100, scale=0.2, rot_dims=48, mlp=None)]
    cfg = U.make_config(layers, width=64, vocab=29, loop=(0, 2, 2), softcap=30.0)
    w = U.random_weights(cfg, seed=31, gain=1.5)
    reqs = [_tokens(cfg, 460, 4), _tokens(cfg, 81, 5)]
    right = [_oracle_logits(cfg, w, t) for t in reqs]
    tol = 3e-2
    for size in (36, 38):  # with a chunk one key off most rows are far over the tolerance
        bad = copy.deepcopy(cfg)
        bad["layers"][0]["mixer"]["mask"]["size"] = size
        assert np.median(_row_err(_oracle_logits(bad, w, reqs[0][:160]), right[0][:160])[44:]) > 2 * tol, size
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
        assert np.median(err) < tol / 2 and np.quantile(err, 0.95) < tol, (np.median(err), err.max())


def test_bf16_chosen_experts(tmp_path):
    # two of eight experts per token, 300 rows (the grouped tensor-core GEMMs) and 60 (the GEMV); a router's close call may come out
    # otherwise at bf16 precision, so most rows are asked for, not all
    cfg = U.make_config([U.gla(heads=2, dim=16, vdim=32, mlp=U.moe(experts=8, top=2, ff=96))], width=64, vocab=29, softcap=30.0)
    w = U.random_weights(cfg, seed=33)
    toks = _tokens(cfg, 300, 6)
    right = _oracle_logits(cfg, w, toks)
    for kw in ({"fault_output_weight": True}, {"fault_renormalised": True}):
        assert np.median(_row_err(_oracle_logits(cfg, w, toks[:60], mlp=kw), right[:60])) > 5e-2, kw
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=40, rows=512)
    whole, cut = _whole(eng, toks), _cuts(eng, toks, [60] * 5)
    eng.close()
    for got in (whole, cut):
        err = _row_err(got, right)
        assert np.median(err) < 1e-2 and np.quantile(err, 0.8) < 2e-2, (np.median(err), err.max())


@pytest.mark.parametrize("width,ff,experts,top,n", [
    (128, 128, 3, 3, 150),   # every expert has every row: a whole tile of rows and a short one
    (160, 136, 2, 2, 200),   # k no multiple of a stage, a tile of output columns that ends early
    (192, 64, 40, 6, 130),   # many experts with few rows each, one stage-wide hidden rows (the down product on the other kernel)
    (256, 320, 5, 1, 700),   # more row tiles than one per expert, two and more tiles of output columns
    (384, 192, 260, 2, 300), # most experts have no row, more of them than a scan's step takes
], ids=["all", "ragged", "many", "tall", "empty_groups"])
def test_bf16_expert_tiles(tmp_path, width, ff, experts, top, n):
    # the grouped expert GEMMs on tcgen05 against the restatement and against portions that take the GEMV; a router's close call may
    # come out otherwise at bf16 precision, so where not every expert is chosen most rows are asked for, not all
    cfg = U.make_config([U.gla(heads=1, dim=8, vdim=8, mlp=U.moe(experts=experts, top=top, ff=ff))], width=width, vocab=29, softcap=30.0)
    w = U.random_weights(cfg, seed=51)
    U.set_values(w, "l0.mlp.router", 0.3 * w["l0.mlp.router"][1])  # scores well below 1, also the best of many
    toks = _tokens(cfg, n, 6)
    right = _oracle_logits(cfg, w, toks)
    assert np.median(_row_err(_oracle_logits(cfg, w, toks[:40], mlp={"fault_output_weight": True}), right[:40])) > 4e-2
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=100, rows=768)
    whole, cut = _whole(eng, toks), _cuts(eng, toks, [n - 33, 1, 32])
    eng.close()
    for got in (whole, cut):
        err = _row_err(got, right)
        assert np.median(err) < 1e-2 and np.quantile(err, 1.0 if top == experts else 0.8) < 2e-2, (np.median(err), err.max())


def test_bf16_other_sizes(tmp_path):
    # bf16 serving precision away from the tensor-core shapes: a width that is no multiple of 64, head sizes beyond the tensor-core
    # kernels' tiles, portions against the whole
    layers = [U.attention(heads=4, kv_heads=2, dim=140, vdim=72, size=50, scale=0.1, rot_dims=10, mlp=U.moe(experts=2, top=2, ff=30)),
              U.gla(heads=3, dim=9, vdim=130), U.gla(heads=1, dim=136, vdim=12)]
    cfg = U.make_config(layers, width=36, vocab=41, softcap=30.0)
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


@pytest.mark.parametrize("dim,vdim,rank,bias,tau", [
    (16, 16, 3, (2.0, 6.0), 16.0),
    (64, 64, 16, (-1.0, 5.0), 16.0),
    (80, 64, 20, (-4.0, 4.0), 2.0),
    (64, 128, 33, (2.0, 8.0), 8.0),
    (128, 96, 8, (-2.0, 3.0), 1.0),
    (20, 12, 5, (-20.0, 3.0), 1.0),    # channels that forget at once beside slow ones: the ranges of a block are too long to factor
    (36, 200, 4, (-2.0, 5.0), 4.0),    # more value columns than a CTA takes
    (64, 24, 4, (-60.0, -40.0), 0.5),  # nothing survives a token
], ids=["small", "square", "padded", "wide_values", "wide_keys", "total_decay_beside_none", "value_blocks", "no_memory"])
def test_bf16_gated_recurrence_in_chunks(tmp_path, dim, vdim, rank, bias, tau):
    # the chunked form at every tile size against the restatement and against the token-by-token form of a copy that is fed in short
    # portions: three sequences in a batch, portions that end inside, at and just behind a chunk of 64
    cfg = U.make_config([U.gla(heads=4, dim=dim, vdim=vdim, tau=tau)], width=64, vocab=29, softcap=30.0)
    w = U.random_weights(cfg, seed=43, rank=rank)
    U.set_values(w, "l0.mix.a2.b", np.random.default_rng(1).uniform(*bias, 4 * dim))
    reqs = [_tokens(cfg, n, 50 + i) for i, n in enumerate([193, 64, 130])]
    right = [_oracle_logits(cfg, w, t) for t in reqs]
    eng = _engine(tmp_path, cfg, w, dtype="bfloat16", page_size=16, max_pages=40, rows=256)
    seqs = [eng.new_sequence() for _ in reqs]
    lg = eng.forward_batch([(seqs[0], reqs[0][:65]), (seqs[1], reqs[1]), (seqs[2], reqs[2][:1])], range(130))
    lg2 = eng.forward_batch([(seqs[2], reqs[2][1:]), (seqs[0], reqs[0][65:192])], range(256))
    lg3 = eng.forward_batch([(seqs[0], reqs[0][192:])], [0])
    steps = _cuts(eng, reqs[2], [2] * 65)
    eng.close()
    got = [np.concatenate([lg[:65], lg2[129:], lg3]), lg[65:129], np.concatenate([lg[129:], lg2[:129]]), steps]
    for g, r in zip(got, right + [right[2]]):
        err = _row_err(g, r)
        assert np.median(err) < 1e-2 and err.max() < 4e-2, (np.median(err), err.max())


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,size,page,rot", [
    (8, 2, 64, 64, 100, 64, 32),    # a tile of keys is one page
    (8, 2, 16, 32, 90, 128, 16),    # a page is two tiles
    (8, 4, 40, 72, 70, 16, 20),     # a head size that takes the fp32 store, padded columns
    (4, 2, 128, 128, 130, 16, 64),  # two blocks of head columns
    (8, 1, 72, 24, 40, 12, 72),     # pages that do not divide a tile: every row by its own address
    (8, 8, 32, 16, 500, 32, 0),     # a chunk longer than the prompt, no rotation
    (4, 4, 8, 200, 64, 16, 0),      # chunk edges on the tiles' edges, more than two blocks of value columns
    (2, 1, 256, 40, 33, 16, 128),   # a head size beyond the tensor-core kernels
    (4, 2, 32, 48, 0, 16, 32),      # no chunks
], ids=["page64", "page128", "fp32_store", "wide_heads", "odd_pages", "one_chunk", "tile_edges", "row_kernel", "causal"])
def test_bf16_prompt_attention_tiles(tmp_path, heads, kv_heads, dim, vdim, size, page, rot):
    # the tensor-core prompt attention (portions of 128 rows and more) against the restatement, and against short portions of the
    # same prompt through the other kernels
    cfg = U.make_config([U.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, size=size, scale=6.0 / dim, rot_dims=rot, base=100.0)], width=64, vocab=29,
                        softcap=30.0)
    w = U.random_weights(cfg, seed=47, gain=1.3)
    toks, other = _tokens(cfg, 300, 9), _tokens(cfg, 140, 10)
    right, right2 = _oracle_logits(cfg, w, toks), _oracle_logits(cfg, w, other)
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

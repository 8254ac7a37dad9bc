"""Kedesun on the CPU: configuration and layer plan, checkpoint reading, the engine's scheduling (portions, mixed batches,
freed pages and slots, generation) against whole sequences of the plain implementation, and that implementation itself."""
import copy
import json
import math

import pytest
import torch

from gcore_b200.models.config import MODEL_ARCH, from_hf_config
from gcore_b200.models.layer_plan import RotarySpec, YarnSpec
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.ops import moe
from gcore_b200.rollout.engine import RolloutWeights, SamplingParams
from tests import kedesun_util as ku
from tests.oracle import kedesun as oracle


# ---------------------------------------------------------------------------------------------- configuration, loading
def test_config_is_read_layer_by_layer():
    c = ku.uneven_conf()
    cfg = from_hf_config(json.loads(json.dumps(c)))
    assert cfg.arch == "kedesun" and cfg.arch in MODEL_ARCH and cfg.vocab_size == 75 and cfg.hidden_size == 44
    assert cfg.tie_word_embeddings and cfg.rms_norm_eps == 1e-5
    a, b, _, d = cfg.layer_plan.layers[:4]
    assert (a.mixer.heads, a.mixer.kv_rank, a.mixer.rot.base, a.mixer.scale) == (3, 36, 500.0, 0.3)
    assert a.mixer.rot.scaling == YarnSpec(3.0, 60, 9.0, 2.0) and (a.ffn.experts, a.ffn.top, a.ffn.shared_ff) == (5, 2, 28)
    assert b.ffn is None and (d.mixer.decay, d.mixer.dim, d.mixer.vdim) == ((0.93,), 40, 70)
    assert [r.layer for r in cfg.layer_plan.runs] == list(range(6))
    assert cfg.num_parameters() == sum(t.numel() for t in oracle.random_weights(c).values())


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Unknown"), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].pop("kv_rank"), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][2]["mlp"].update(kind="other"), lambda c: c["layers"][3]["mixer"].update(decay=[0.5, 0.5]),
    lambda c: c["layers"][3]["mixer"].update(decay=[1.5]), lambda c: c["layers"][0]["mlp"]["router"].update(top=6),
    lambda c: c.update(layers=[])])
def test_what_the_design_does_not_have_is_refused(edit):
    c = copy.deepcopy(ku.uneven_conf())
    edit(c)
    with pytest.raises((ValueError, KeyError)):
        from_hf_config(c)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (6, 500.0, 3.0, 60, 9.0, 2.0), (64, 10000.0, 40.0, 4096, 32.0, 1.0), (2, 100.0, 2.0, 10, 1.0, 1.0),
    (16, 50.0, 8.0, 16, 4.0, 4.0), (8, 10.0, 0.5, 100000, 64.0, 0.5)])
def test_rotation_frequencies(dims, base, factor, original, fast, slow):
    """Against the plain implementation, and the limits by hand: fast pairs keep their frequency, slow ones are divided."""
    spec = RotarySpec(dims, base, YarnSpec(factor, original, fast, slow))
    rot = ku.rotation(dims, base, factor, original, fast, slow)
    f, m = oracle.frequencies(rot)
    assert spec.frequencies() == pytest.approx(f, rel=1e-14) and spec.magnitude() == pytest.approx(m)
    assert m == pytest.approx(0.1 * math.log(factor) + 1)
    plain = RotarySpec(dims, base)
    assert plain.magnitude() == 1.0 and plain.frequencies() == [base ** (-2 * i / dims) for i in range(dims // 2)]
    for i, (a, b) in enumerate(zip(f, plain.frequencies())):
        lo, hi = sorted((b, b / factor))
        assert lo * (1 - 1e-12) <= a <= hi * (1 + 1e-12)


def test_checkpoint_tensors_must_fit_exactly():
    c = ku.uneven_conf()
    W = oracle.random_weights(c)
    cfg = from_hf_config(c)
    for bad in ({k: v for k, v in W.items() if k != "l0.mlp.e3.down"}, {**W, "l1.mlp.gate": W["l2.mlp.gate"]},
                {**W, "l0.mix.o": W["l0.mix.o"][:, :-1]}, {**W, "l3.dwa": W["l3.dwa"][:-1]}):
        with pytest.raises((KeyError, ValueError)):
            build_decoder(cfg).load_tensors(bad)
    m = build_decoder(cfg).load_tensors(W)
    mix = m.layers[0].mixer       # padded heads: real rows in place, zero rows between them
    ly = mix.layout
    q = m.layers[0].in_proj[:3 * (ly.dim + ly.row_rot)].view(3, ly.dim + ly.row_rot, -1)
    want = W["l0.mix.q"].view(3, 26, 44)
    assert torch.equal(q[:, :20, :44], want[:, :20]) and torch.equal(q[:, ly.dim:ly.dim + 6, :44], want[:, 20:])
    assert not q[:, 20:ly.dim].any() and not q[:, ly.dim + 6:].any() and not q[..., 44:].any()
    assert m.output_weight is m.embed


def test_layers_ask_for_the_cache_and_state_they_use():
    c = ku.uneven_conf()
    eng = ku.make_engine(c, oracle.random_weights(c), max_model_len=32)
    eng.wake_up()
    kinds = [sp["type"] for sp in c["layers"]]
    assert [x is not None for x in eng.k_cache] == [k == "latent_attention" for k in kinds]
    assert [x is not None for x in eng.memory] == [k == "retention" for k in kinds]
    rows = sum(x.shape[-1] for x in eng.k_cache if x is not None)
    assert eng._kv_bytes_per_block() == rows * eng.bs * 4
    assert eng.plan.state_bytes_per_slot() == sum(4 * x.S[0].numel() for x in eng.memory if x is not None)


def test_registered_and_served_only():
    from gcore_b200 import build_native
    from gcore_b200.models.config import build_model_config
    from gcore_b200.models.gpt import GPTModel
    from gcore_b200.ops import registry
    c = ku.uneven_conf()
    assert build_model_config("kedesun", {"hf_config": c}).layer_plan == from_hf_config(c).layer_plan
    with pytest.raises(ValueError, match="config.json"):
        build_model_config("kedesun")
    with pytest.raises(ValueError, match="served"):
        GPTModel(from_hf_config(c))
    eng = ku.make_engine(c, oracle.random_weights(c), max_model_len=32)
    with pytest.raises(NotImplementedError):
        eng.quantize_weights_fp8()
    assert {"latent_attention", "retention", "routed_experts", "add_layer"} <= set(registry.available())
    assert all((build_native.OPS_SRC / f"{s}.cu").exists() for s in build_native.KERNEL_SETS["kedesun"])
    with pytest.raises(ValueError, match="experts"):
        build_decoder(from_hf_config(ku.conf([ku.retention(1, 8, 8, ku.experts(513, 2, 8, 8))], 8, 16)))


def test_new_weights_replace_the_old_ones():
    c = ku.uneven_conf()
    Wa, Wb = oracle.random_weights(c, seed=1), oracle.random_weights(c, seed=2)
    eng = ku.make_engine(c, Wa, max_model_len=64)
    seq = ku.tokens(20, 75, 1)
    eng.update_weights(RolloutWeights.from_model(build_decoder(eng.cfg).load_tensors(Wb)))
    ku.assert_close(ku.run_alone(eng, seq, [20]), oracle.forward(Wb, c, seq))
    eng.load_weights_from(build_decoder(eng.cfg).load_tensors(Wa))
    ku.assert_close(ku.run_alone(eng, seq, [20]), oracle.forward(Wa, c, seq))


# --------------------------------------------------------------------------------------------------------- plain oracle
def test_plain_rotation_turns_neighbours_and_keeps_distances():
    rot = ku.rotation(6, 50.0, factor=2.0, original=40, fast=4.0, slow=1.0)
    torch.manual_seed(0)
    q, k = torch.randn(1, 6).double(), torch.randn(1, 6).double()
    m2 = oracle.frequencies(rot)[1] ** 2
    at = lambda x, p: oracle.rotate(x, rot, [p])[0]
    assert float(at(q, 0) @ at(k, 0)) == pytest.approx(m2 * float(q[0] @ k[0]))
    assert float(at(q, 9) @ at(k, 4)) == pytest.approx(float(at(q, 905) @ at(k, 900)))    # only the distance counts
    one = torch.zeros(1, 6).double()
    one[0, 2] = 1.0                                                                       # second pair, first element
    y = oracle.rotate(one, dict(dims=6, base=50.0), [3])[0]
    a = 3 * 50.0 ** (-2 / 6)
    assert y[2] == pytest.approx(math.cos(a)) and y[3] == pytest.approx(math.sin(a)) and y[[0, 1, 4, 5]].abs().sum() == 0


def test_plain_retention_matches_its_sum_form():
    """The recurrence = the plain double sum with powers of the decay, with and without a carried state."""
    torch.manual_seed(0)
    q, k, v = torch.randn(11, 2, 3).double(), torch.randn(11, 2, 3).double(), torch.randn(11, 2, 5).double()
    decay = [0.8, 1.0]
    whole = oracle.retention_core(q, k, v, decay)
    S = torch.zeros(2, 3, 5).double()
    parts = torch.cat([oracle.retention_core(q[a:b], k[a:b], v[a:b], decay, S) for a, b in ((0, 4), (4, 5), (5, 11))])
    assert (whole - parts).abs().max() < 1e-12
    for t in range(11):
        for a in range(2):
            want = sum(decay[a] ** (t - s) * (q[t, a] @ k[s, a]) * 3 ** -0.5 * v[s, a] for s in range(t + 1))
            assert (whole[t, a] - want).abs().max() < 1e-12


def test_plain_choice_uses_the_correction_for_the_choice_only():
    z, corr = torch.tensor([2.0, 1.0, 0.0, -1.0]).double(), torch.tensor([0.0, 0.0, 5.0, 0.0]).double()
    s = torch.softmax(z, 0)
    got = dict(oracle.choose_experts(z, corr, 2))
    assert set(got) == {0, 2} and got[0] == pytest.approx(float(s[0] / (s[0] + s[2])))


def test_plain_depth_average_by_hand():
    """Two layers that add nothing: the stream is a product of the averages' weights."""
    c = ku.conf([ku.retention(1, 4, 4, None), ku.retention(1, 4, 4, None)], 8, 11)
    W = oracle.random_weights(c)
    for i in (0, 1):
        W[f"l{i}.mix.o"] = torch.zeros_like(W[f"l{i}.mix.o"])
    W["l0.dwa"], W["l1.dwa"] = torch.tensor([0.5, 0.25]), torch.tensor([1.0, 2.0, 4.0])
    seen = []
    oracle.forward(W, c, [3], collect=seen)
    e = W["embed"][3].double()
    assert torch.allclose(seen[0][0], 0.75 * e) and torch.allclose(seen[1][0], (1 + 2 + 4 * 0.75) * e)


@pytest.mark.parametrize("fault", ["decay", "scale", "pairs", "magnitude", "ramp", "gate", "latent norm", "average", "correction",
                                   "shared gate", "silu", "eps", "norms"])
def test_a_planted_mistake_shows(fault, monkeypatch):
    """The test models are sensitive: one wrong piece in the plain implementation moves the logits far beyond rounding."""
    c = ku.uneven_conf()
    W = oracle.random_weights(c, seed=2)
    seq = ku.tokens(60, 75, 3)
    eng = ku.make_engine(c, W, max_model_len=128)
    got = ku.run_alone(eng, seq, [60])
    ku.assert_close(got, oracle.forward(W, c, seq))
    bad, Wb = copy.deepcopy(c), dict(W)
    if fault == "decay":
        bad["layers"][3]["mixer"]["decay"] = [0.9]
    elif fault == "scale":
        bad["layers"][2]["mixer"]["scale"] *= 1.1
    elif fault == "pairs":        # halves in place of neighbours
        right = oracle.rotate
        mix = lambda x, n: torch.cat([x[..., 0:n:2], x[..., 1:n:2]], -1)
        monkeypatch.setattr(oracle, "rotate", lambda x, rot, p: right(mix(x, rot["dims"]), rot, p))
    elif fault in ("magnitude", "ramp"):
        right_f = oracle.frequencies
        monkeypatch.setattr(oracle, "frequencies", lambda rot: (right_f(rot)[0], 1.0) if fault == "magnitude" else
                            ([f / 2 for f in right_f(rot)[0]], right_f(rot)[1]))
    elif fault == "gate":
        for i in (0, 2, 4):
            Wb[f"l{i}.mix.g"] = torch.zeros_like(W[f"l{i}.mix.g"])
    elif fault == "latent norm":
        Wb["l0.mix.dkv.norm"] = torch.ones_like(W["l0.mix.dkv.norm"])
    elif fault == "average":
        monkeypatch.setattr(oracle, "depth_average", lambda w, r: sum(a * x for a, x in zip(w.flip(0), r)))
    elif fault == "correction":
        Wb["l0.mlp.correction"] = torch.zeros_like(W["l0.mlp.correction"])
    elif fault == "shared gate":
        Wb["l3.mlp.shared.sg"] = torch.zeros_like(W["l3.mlp.shared.sg"])
    elif fault == "silu":
        monkeypatch.setattr(oracle, "silu", torch.relu)
    elif fault == "norms":
        monkeypatch.setattr(oracle, "rms", lambda x, eps: x)
    else:
        bad["norm"]["eps"] = 1e-1
    assert ku.rms_error(got, oracle.forward(Wb, bad, seq)).max() > 1e-2


# --------------------------------------------------------------------------------------------------------------- engine
def test_portions_match_the_whole_prompt():
    c = ku.uneven_conf()
    W = oracle.random_weights(c, seed=4)
    eng = ku.make_engine(c, W, max_model_len=128, kv_block_size=8)
    for n in (1, 2, 39, 77):
        seq = ku.tokens(n, 75, n)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [7, 1, 3], [36, 2, 1]):
            ku.assert_close(ku.run_alone(eng, seq, cuts), want, what=(n, cuts))
    st = eng.get_load()
    assert st["free_blocks"] == st["num_blocks"] and st["running"] == 0


def test_stream_after_every_layer():
    c = ku.uneven_conf()
    W = oracle.random_weights(c, seed=5)
    eng = ku.make_engine(c, W, max_model_len=64)
    eng.wake_up()
    seq, want, got = ku.tokens(17, 75, 9), [], []
    oracle.forward(W, c, seq, collect=want)
    rid = eng.open_request()
    assert eng.sched.reserve(rid, 17) == 0
    rows, _ = eng._step_rows([(rid, 0, seq)])
    eng.plan(rows, eng.k_cache, eng.memory, record=got)
    for g, w in zip(got, want):
        assert (g[:, :44] - w).abs().max() < 1e-4 * w.abs().max()


def test_mixed_requests_on_a_small_pool():
    """Nine requests through four slots and a pool that only holds four: pages and slots are used again."""
    c = ku.uneven_conf()
    W = oracle.random_weights(c, seed=5)
    eng = ku.make_engine(c, W, max_model_len=64, kv_block_size=4, num_kv_blocks=48)
    seqs = [ku.tokens(n, 75, 60 + n) for n in (40, 7, 21, 1, 44, 13, 30, 2, 39)]
    for s, got in zip(seqs, ku.run_mixed(eng, seqs, [1, 1, 2, 5, 9, 17], seed=1)):
        ku.assert_close(got, oracle.forward(W, c, s))
    assert eng.get_load()["free_blocks"] == 48


@pytest.mark.parametrize("kind", ["retention", "latent"])
def test_plans_of_one_kind_of_mixer(kind):
    """No cache at all, or no state at all."""
    ly = [ku.retention(2, 12, 10, ku.dense(20)) if kind == "retention" else ku.latent(2, 12, 4, 10, 20, 0.3, ku.dense(20))] * 2
    c = ku.conf(ly, 24, 40)
    W = oracle.random_weights(c, seed=6)
    eng = ku.make_engine(c, W, max_model_len=64, kv_block_size=8)
    seq = ku.tokens(30, 40, 1)
    ku.assert_close(ku.run_alone(eng, seq, [11, 1, 2]), oracle.forward(W, c, seq))
    a, b = eng.generate([seq[:9]], SamplingParams(max_new_tokens=8, greedy=True), n=2)
    assert a.out_tokens == b.out_tokens == _greedy(W, c, seq[:9], 8)


def _greedy(W, c, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(oracle.forward(W, c, t)[-1].argmax()))
    return t[len(prompt):]


def test_greedy_generation_with_shared_prompts_and_stops():
    c = ku.uneven_conf()
    W = oracle.random_weights(c, seed=6)
    eng = ku.make_engine(c, W, max_model_len=48, kv_block_size=4, max_prefill_tokens=6, sync_interval=4)
    prompts = [ku.tokens(n, 75, 80 + n) for n in (1, 4, 9, 15)]
    want = [_greedy(W, c, p, 8) for p in prompts]
    for k, r in enumerate(eng.generate(prompts, SamplingParams(max_new_tokens=8, greedy=True), n=2)):
        assert r.out_tokens == want[k // 2] and r.finish_reason == "length"
    stop = want[0][3]
    for w, r in zip(want, eng.generate(prompts, SamplingParams(max_new_tokens=8, greedy=True, stop_token_ids=(stop,)))):
        assert r.out_tokens == (w[:w.index(stop) + 1] if stop in w else w)
    assert eng.get_load()["free_blocks"] == eng.num_blocks
    eng.sleep()
    assert not eng.memory and not eng.k_cache
    assert eng.generate(prompts[:1], SamplingParams(max_new_tokens=8, greedy=True))[0].out_tokens == want[0]


def test_sampling_is_per_request_and_reproducible():
    c = ku.uneven_conf()
    eng = ku.make_engine(c, oracle.random_weights(c, seed=7), max_model_len=32)
    runs = [eng.generate([[5, 6, 7]], SamplingParams(max_new_tokens=6, seed=3, temperature=3.0), n=4) for _ in range(2)]
    assert [r.out_tokens for r in runs[0]] == [r.out_tokens for r in runs[1]]
    assert len({tuple(r.out_tokens) for r in runs[0]}) > 1


def test_expert_segments_never_overlap():
    torch.manual_seed(1)
    for T, E, K in ((1, 1, 1), (3, 200, 16), (40, 5, 2), (300, 2, 2)):
        counts = torch.zeros(E, dtype=torch.int32)
        idx, w, place = moe.choose(torch.randn(T, E + 1), E, K, torch.randn(E), counts)
        assert int(counts.sum()) == T * K and torch.allclose(w.sum(-1), torch.ones(T))
        h = torch.randn(T, 8)
        rows, dest, off = moe.expert_rows(h, counts, idx, place)
        assert dest.unique().numel() == T * K and int(off[-1]) <= rows.shape[0] and not (off % moe.SEG).any()
        assert ((dest >= off[idx]) & (dest < off[idx] + counts[idx])).all()
        assert torch.equal(rows[dest.long()], h[:, None].expand(-1, K, -1))

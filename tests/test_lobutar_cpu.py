"""Lobutar on the CPU: configuration and layer plan, checkpoint reading, the engine's scheduling (portions, mixed batches,
freed pages and slots, generation) against whole sequences of the plain implementation, and that implementation itself."""
import copy
import json
import math

import pytest
import torch

from gcore_b200.models.config import MODEL_ARCH, from_hf_config
from gcore_b200.models.layer_plan import LayerPlan
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.ops import moe
from gcore_b200.ops.rows import portion_contexts
from gcore_b200.rollout.engine import RolloutWeights, SamplingParams
from tests import lobutar_util as lu
from tests.oracle import lobutar as oracle


# ---------------------------------------------------------------------------------------------- configuration, loading
def test_config_is_read_layer_by_layer():
    c = lu.uneven_conf()
    cfg = from_hf_config(json.loads(json.dumps(c)))
    assert cfg.arch == "lobutar" and cfg.arch in MODEL_ARCH and cfg.vocab_size == 75 and cfg.hidden_size == 44
    assert not cfg.tie_word_embeddings and cfg.rms_norm_eps == 1e-5 and cfg.num_layers == 9
    plan = cfg.layer_plan
    assert plan.streams == 3 and plan.names == (0, 1, 2, 3, 5, 6) and plan.windows() == [1, 9, 70]
    assert [r.layer for r in plan.runs] == [0, 1, 2, 3, 0, 4, 5, 0, 5] and [r.index for r in plan.runs] == list(range(9))
    a, b, d, e = plan.layers[:4]
    assert (a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim, a.mixer.rot.dims) == (6, 2, 20, 12, 6)
    assert (a.mixer.scale, a.mixer.diff, d.mixer.rot.base, d.ffn) == (0.3, 0.2, 90.0, None)
    assert (b.mixer.window, b.mixer.sink, b.mixer.gate, b.mixer.kv_rank) == (9, True, "element", 36)
    assert (a.ffn.groups, a.ffn.keep, a.ffn.scale, a.ffn.score, a.ffn.normalize, a.ffn.act) == (3, 2, 2.5, "sigmoid", False,
                                                                                              "silu_gate")
    assert (e.ffn.shared_ff, e.ffn.groups, e.ffn.shared_gate) == (0, 1, False)
    assert cfg.num_parameters() == sum(t.numel() for t in oracle.random_weights(c).values())


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Unknown"), lambda c: c["layers"][0].update(type="other"), lambda c: c.update(layers=[]),
    lambda c: c["layers"][1]["mixer"].pop("kv_rank"), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][1]["mixer"].pop("mask"), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=4), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22),
    lambda c: c["layers"][0]["mixer"].pop("diff"), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), lambda c: c["layers"][1]["mlp"].update(kind="other"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c.pop("streams"), lambda c: c.update(streams=0),
    lambda c: c["layers"][4].update(weights_of=9), lambda c: c["layers"][0].update(weights_of=4)])
def test_what_the_design_does_not_have_is_refused(edit):
    c = copy.deepcopy(lu.uneven_conf())
    edit(c)
    with pytest.raises((ValueError, KeyError)):
        from_hf_config(c)


def test_layers_may_borrow_from_later_ones_and_through_others():
    c = lu.uneven_conf()
    ly = [dict(c["layers"][1]), c["layers"][0], c["layers"][1], dict(c["layers"][1])]
    ly[0]["weights_of"], ly[3]["weights_of"] = 2, 0
    plan = from_hf_config(dict(c, layers=ly)).layer_plan
    assert plan.names == (1, 2) and plan.order == (1, 0, 1, 1)
    with pytest.raises(ValueError):
        LayerPlan(plan.layers, order=(0, 2))
    with pytest.raises(ValueError):
        LayerPlan(plan.layers, names=(0,))


def test_checkpoint_tensors_must_fit_exactly():
    c = lu.uneven_conf()
    W = oracle.random_weights(c)
    cfg = from_hf_config(c)
    for bad in ({k: v for k, v in W.items() if k != "l0.mlp.e3.down"}, {**W, "l4.norm1": W["l0.norm1"]},
                {**W, "l0.mix.o": W["l0.mix.o"][:, :-1]}, {**W, "l3.hc1.mix": W["l3.hc1.mix"][:-1]},
                {k: v for k, v in W.items() if k != "l1.mix.sink"}, {k: v for k, v in W.items() if k != "l2.mix.v.b"}):
        with pytest.raises((KeyError, ValueError)):
            build_decoder(cfg).load_tensors(bad)
    m = build_decoder(cfg).load_tensors(W)
    sub = m.layers[0].mixer       # padded heads: real rows in place, zero rows between them
    ly = sub.part.layout
    k = sub.in_proj[ly.k:ly.k + 4 * ly.dim].view(4, ly.dim, -1)
    assert torch.equal(k[:, :20, :44], W["l0.mix.k"].view(4, 20, 44)) and not k[:, 20:].any() and not k[..., 44:].any()
    b = sub.in_bias[ly.v:ly.v + 2 * ly.vdim].view(2, ly.vdim)
    assert torch.equal(b[:, :12], W["l0.mix.v.b"].view(2, 12).float()) and not b[:, 12:].any()
    assert not sub.in_bias[ly.gate:].any() and torch.equal(sub.out_bias[:44], W["l0.mix.o.b"].float())
    m.load_tensors({**W, "l2.norm2": torch.zeros(3), "l6.hc2.mix": torch.zeros(1)})    # no feed-forward: nothing reads them


def test_layers_ask_for_the_cache_they_use():
    c = lu.uneven_conf()
    eng = lu.make_engine(c, oracle.random_weights(c), max_model_len=32)
    eng.wake_up()
    assert len(eng.k_cache) == 9 and len({x.data_ptr() for x in eng.k_cache}) == 9      # one per run, shared weights or not
    assert eng.k_cache[0].shape == eng.k_cache[4].shape == eng.k_cache[7].shape
    assert eng.k_cache[2].shape[2] == 3 * 2 * 16 + 3 * 32 and all(x is None for x in eng.memory)
    rows = sum(x[0, 0].numel() for x in eng.k_cache)
    assert eng._kv_bytes_per_block() == rows * eng.bs * 4 and eng.plan.state_bytes_per_slot() == 0


def test_registered_and_served_only():
    from gcore_b200 import build_native
    from gcore_b200.models.config import build_model_config
    from gcore_b200.models.gpt import GPTModel
    from gcore_b200.ops import registry
    c = lu.uneven_conf()
    assert build_model_config("lobutar", {"hf_config": c}).layer_plan == from_hf_config(c).layer_plan
    with pytest.raises(ValueError, match="config.json"):
        build_model_config("lobutar")
    with pytest.raises(ValueError, match="served"):
        GPTModel(from_hf_config(c))
    eng = lu.make_engine(c, oracle.random_weights(c), max_model_len=32)
    with pytest.raises(NotImplementedError):
        eng.quantize_weights_fp8()
    assert {"latent_attention", "differential_attention", "connect", "routed_experts"} <= set(registry.available())
    assert all((build_native.OPS_SRC / f"{s}.cu").exists() for s in build_native.KERNEL_SETS["lobutar"])
    one = lu.latent(1, 8, 4, 8, 8, 4, 0.2, None)
    with pytest.raises(ValueError, match="experts"):
        build_decoder(from_hf_config(lu.conf([dict(one, mlp=lu.experts(513, 2, 8, 8))], 8, 16)))
    with pytest.raises(ValueError, match="groups"):
        build_decoder(from_hf_config(lu.conf([dict(one, mlp=lu.experts(66, 2, 8, 8, groups=33, keep=4))], 8, 16)))
    with pytest.raises(ValueError, match="streams"):
        build_decoder(from_hf_config(lu.conf([one], 8, 16, streams=17)))


def test_new_weights_replace_the_old_ones():
    c = lu.uneven_conf()
    Wa, Wb = oracle.random_weights(c, seed=1), oracle.random_weights(c, seed=2)
    eng = lu.make_engine(c, Wa, max_model_len=64)
    seq = lu.tokens(20, 75, 1)
    eng.update_weights(RolloutWeights.from_model(build_decoder(eng.cfg).load_tensors(Wb)))
    lu.assert_close(lu.run_alone(eng, seq, [20]), oracle.forward(Wb, c, seq))
    eng.load_weights_from(build_decoder(eng.cfg).load_tensors(Wa))
    lu.assert_close(lu.run_alone(eng, seq, [20]), oracle.forward(Wa, c, seq))


def test_portion_contexts_hold_what_a_window_sees():
    start, cu, n, before = portion_contexts([0, 5, 40], [3, 2, 10], 8)
    assert start.tolist() == [0, 0, 33] and cu.tolist() == [0, 3, 10, 27] and (n, before) == (27, 7)
    start, cu, n, before = portion_contexts([0, 5, 40], [3, 2, 10], 0)
    assert start.tolist() == [0, 0, 0] and cu.tolist() == [0, 3, 10, 60] and (n, before) == (60, 40)
    assert portion_contexts([], [], 8)[2:] == (0, 0) and portion_contexts([9], [4], 1)[0].tolist() == [9]


# --------------------------------------------------------------------------------------------------------- plain oracle
def test_plain_rotation_turns_leading_neighbours_and_keeps_distances():
    rot = lu.rotation(4, 50.0)
    torch.manual_seed(0)
    q, k = torch.randn(1, 6).double(), torch.randn(1, 6).double()
    at = lambda x, p: oracle.rotate(x, rot, [p])[0]
    assert float(at(q, 9) @ at(k, 4)) == pytest.approx(float(at(q, 905) @ at(k, 900)))    # only the distance counts
    assert torch.equal(at(q, 7)[4:], q[0, 4:])
    one = torch.zeros(1, 6).double()
    one[0, 2] = 1.0                                                                       # second pair, first element
    y, a = at(one, 3), 3 * 50.0 ** (-2 / 4)
    assert y[2] == pytest.approx(math.cos(a)) and y[3] == pytest.approx(math.sin(a)) and y[[0, 1, 4, 5]].abs().sum() == 0


def test_plain_window_and_sink_by_hand():
    assert list(oracle.visible(5)) == [0, 1, 2, 3, 4, 5] and list(oracle.visible(5, 1)) == [5]
    assert list(oracle.visible(5, 3)) == [3, 4, 5] and list(oracle.visible(1, 3)) == [0, 1]
    w = oracle.softmax_with_sink(torch.zeros(3).double(), torch.tensor(math.log(2.0)).double())
    assert torch.allclose(w, torch.full((3,), 0.2).double())                              # 1 + 1 + 1 and 2 for the sink
    s = torch.tensor([700.0, 701.0]).double()
    assert oracle.softmax_with_sink(s, torch.tensor(900.0).double()).max() < 1e-80        # no overflow either way
    assert torch.allclose(oracle.softmax_with_sink(s, torch.tensor(-900.0).double()), torch.softmax(s, 0))


def test_plain_difference_of_maps_by_hand():
    z = torch.zeros(2).double()
    assert oracle.difference_weight(z, z, z, z, 0.3) == pytest.approx(0.3)
    one = torch.ones(2).double()
    assert oracle.difference_weight(one, one, z, one, 0.1) == pytest.approx(math.e ** 2 - 1 + 0.1)
    o = oracle.combine_maps(torch.tensor([[3.0, 4.0]]).double(), torch.tensor([[2.0, 0.0]]).double(), 1.5, 0.25, 0.0)
    assert torch.allclose(o, torch.tensor([[0.0, 0.75 * 2 ** 0.5]]).double())             # (0, 4) normed, times 3/4


def test_plain_choice_keeps_the_best_groups_and_the_bare_scores():
    z = torch.tensor([4.0, -4.0, 1.0, 1.0, 0.5, 0.5, -1.0, 9.0]).double()
    corr = torch.tensor([-2.0, -2.0, -2.0, -2.0, -2.0, -2.0, -2.0, -9.0]).double()        # every choice score is negative
    router = dict(top=2, scale=3.0, groups=dict(count=4, keep=1))
    s = torch.sigmoid(z)
    got = dict(oracle.choose_experts(z, corr, router))                                    # 0 alone is better, 2 + 3 is not
    assert set(got) == {2, 3} and got[2] == pytest.approx(3 * float(s[2]))
    assert set(dict(oracle.choose_experts(z, corr, dict(top=2)))) == {0, 2}
    flat = torch.zeros(8).double()
    assert set(dict(oracle.choose_experts(z, flat, dict(top=1, groups=dict(count=8, keep=1))))) == {7}


def test_plain_streams_by_hand():
    x = torch.tensor([1.0, 10.0]).double().view(2, 1, 1)
    mix, out, y = torch.tensor([[1.0, 2.0], [3.0, 4.0]]).double(), torch.tensor([5.0, 6.0]).double(), torch.full((1, 1), 100.0)
    new = oracle.write_streams(mix, out, x, y.double())                                   # [from, to], from the old ones
    assert new.flatten().tolist() == [1 + 30 + 500, 2 + 40 + 600]
    assert float(oracle.read_streams(out, x)) == 65.0


@pytest.mark.parametrize("fault", ["window", "sink", "pairs", "dims", "scale", "diff", "lambda", "second map", "map order",
                                   "head gate", "element gate", "biases", "output bias", "latent norm", "mix order", "read",
                                   "write", "stream sum", "correction", "groups", "masked as zero", "router scale", "normalised",
                                   "shared", "silu", "eps", "norms", "run once"])
def test_a_planted_mistake_shows(fault, monkeypatch):
    """The test models are sensitive: one wrong piece in the plain implementation moves the logits far beyond rounding."""
    c = lu.uneven_conf()
    W = oracle.random_weights(c, seed=2)
    if fault == "masked as zero":      # matters where choice scores are negative
        for i in (0, 3):
            W[f"l{i}.mlp.correction"] = W[f"l{i}.mlp.correction"] - 2
    seq = lu.tokens(60, 75, 3)
    eng = lu.make_engine(c, W, max_model_len=128)
    got = lu.run_alone(eng, seq, [60])
    lu.assert_close(got, oracle.forward(W, c, seq))
    bad, Wb = json.loads(json.dumps(c)), dict(W)
    zero = lambda end: Wb.update({k: torch.zeros_like(v) for k, v in W.items() if k.endswith(end)})
    mixers = lambda kind: [sp["mixer"] for sp in bad["layers"] if sp["type"] == kind]
    routers = [sp["mlp"]["router"] for sp in bad["layers"] if sp["mlp"] and sp["mlp"]["kind"] == "moe"]
    if fault == "window":
        for m in mixers("latent_attention"):
            m["mask"]["size"] += 1
    elif fault == "sink":
        Wb.update({k: v - 50 for k, v in W.items() if k.endswith(".sink")})
    elif fault == "pairs":             # halves in place of neighbours
        right = oracle.rotate
        halves = lambda x, n: torch.cat([x[..., 0:n:2], x[..., 1:n:2], x[..., n:]], -1)
        monkeypatch.setattr(oracle, "rotate", lambda x, rot, p: right(halves(x, rot["dims"]), rot, p))
    elif fault == "dims":
        bad["layers"][0]["mixer"]["rot"]["dims"] += 2
    elif fault == "scale":
        for m in mixers("attention"):
            m["scale"] *= 1.1
    elif fault == "diff":
        right_c = oracle.combine_maps
        monkeypatch.setattr(oracle, "combine_maps", lambda a1, a2, lam, diff, eps: right_c(a1, a2, lam, 0.0, eps))
    elif fault == "lambda":
        monkeypatch.setattr(oracle, "difference_weight", lambda *a: a[-1])
    elif fault == "second map":
        monkeypatch.setattr(oracle, "combine_maps", lambda a1, a2, lam, diff, eps: oracle.rms(a1, eps) * (1 - diff))
    elif fault == "map order":
        right_c = oracle.combine_maps
        monkeypatch.setattr(oracle, "combine_maps", lambda a1, a2, *a: right_c(a2, a1, *a))
    elif fault == "head gate":
        zero("l0.mix.g")
    elif fault == "element gate":
        zero("l1.mix.g")
    elif fault == "biases":
        zero("mix.v.b")
    elif fault == "output bias":
        zero("mix.o.b")
    elif fault == "latent norm":
        Wb["l1.mix.dkv.norm"] = torch.ones_like(W["l1.mix.dkv.norm"])
    elif fault == "mix order":
        Wb.update({k: v.T.contiguous() for k, v in W.items() if ".hc" in k and k.endswith(".mix")})
    elif fault == "read":
        Wb.update({k: torch.full_like(v, 1 / 3) for k, v in W.items() if k.endswith("hc2.in")})
    elif fault == "write":
        Wb.update({k: torch.ones_like(v) for k, v in W.items() if k.endswith("hc1.out")})
    elif fault == "stream sum":        # every stream's share of the end result
        right_s = oracle.sublayer
        monkeypatch.setattr(oracle, "sublayer", lambda W, n, q, x, eps, run: right_s(W, n, q, x, eps, run) if n != "l6" else
                            right_s(W, n, q, x, eps, run) * torch.tensor([1.0, 1.0, 0.0]).double().view(3, 1, 1))
    elif fault == "correction":
        zero("correction")
    elif fault == "groups":
        for r in routers:
            r.pop("groups")
    elif fault == "masked as zero":
        def choose(z, corr, r):
            n, s = len(z) // r["groups"]["count"], torch.sigmoid(z)
            ch = [float(s[e] + corr[e]) for e in range(len(z))]
            gs = [sum(sorted(ch[g * n:(g + 1) * n])[-2:]) for g in range(r["groups"]["count"])]
            kept = sorted(range(len(gs)), key=lambda g: -gs[g])[:r["groups"]["keep"]]
            best = sorted(range(len(z)), key=lambda e: -(ch[e] if e // n in kept else 0.0))[:r["top"]]
            return [(e, float(s[e]) * r["scale"]) for e in best]
        monkeypatch.setattr(oracle, "choose_experts", choose)
    elif fault == "router scale":
        for r in routers:
            r["scale"] = 1.0
    elif fault == "normalised":
        right_r = oracle.choose_experts
        monkeypatch.setattr(oracle, "choose_experts", lambda *a: (lambda p: [(e, w / sum(x for _, x in p)) for e, w in p])(
            right_r(*a)))
    elif fault == "shared":
        zero("shared.down")
    elif fault == "silu":
        monkeypatch.setattr(oracle, "silu", torch.relu)
    elif fault == "norms":
        monkeypatch.setattr(oracle, "rms", lambda x, eps: x)
    elif fault == "run once":          # a layer that comes back runs again
        right_l, seen = oracle.layer, set()
        monkeypatch.setattr(oracle, "layer", lambda W, n, sp, x, eps: x if n in seen or seen.add(n) else
                            right_l(W, n, sp, x, eps))
    else:
        bad["norm"]["eps"] = 1e-1
    assert lu.rms_error(got, oracle.forward(Wb, bad, seq)).max() > 1e-2


# --------------------------------------------------------------------------------------------------------------- engine
def test_portions_match_the_whole_prompt():
    c = lu.uneven_conf()
    W = oracle.random_weights(c, seed=4)
    eng = lu.make_engine(c, W, max_model_len=128, kv_block_size=8)
    for n in (1, 2, 39, 77):
        seq = lu.tokens(n, 75, n)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [7, 1, 3], [36, 2, 1]):
            lu.assert_close(lu.run_alone(eng, seq, cuts), want, what=(n, cuts))
    st = eng.get_load()
    assert st["free_blocks"] == st["num_blocks"] and st["running"] == 0


@pytest.mark.parametrize("streams", [1, 2, 5])
def test_residual_after_every_layer(streams):
    c = dict(lu.uneven_conf(), streams=streams)
    W = oracle.random_weights(c, seed=5)
    eng = lu.make_engine(c, W, max_model_len=64)
    eng.wake_up()
    seq, want, got = lu.tokens(17, 75, 9), [], []
    oracle.forward(W, c, seq, collect=want)
    rid = eng.open_request()
    assert eng.sched.reserve(rid, 17) == 0
    rows, _ = eng._step_rows([(rid, 0, seq)])
    eng.plan(rows, eng.k_cache, eng.memory, record=got)
    assert len(got) == len(want) == 9
    for g, w in zip(got, want):
        assert (g[:, :44] - w).abs().max() < 1e-4 * w.abs().max()


def test_mixed_requests_on_a_small_pool():
    """Nine requests through four slots and a pool that only holds four: pages and slots are used again."""
    c = lu.uneven_conf()
    W = oracle.random_weights(c, seed=5)
    eng = lu.make_engine(c, W, max_model_len=64, kv_block_size=4, num_kv_blocks=48)
    seqs = [lu.tokens(n, 75, 60 + n) for n in (40, 7, 21, 1, 44, 13, 30, 2, 39)]
    for s, got in zip(seqs, lu.run_mixed(eng, seqs, [1, 1, 2, 5, 9, 17], seed=1)):
        lu.assert_close(got, oracle.forward(W, c, s))
    assert eng.get_load()["free_blocks"] == 48


def _greedy(W, c, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(oracle.forward(W, c, t)[-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_plans_of_one_kind_of_mixer(kind):
    one = lu.attention(4, 1, 12, 10, 4, 0.3, 0.4, lu.dense(20)) if kind == "attention" else \
        lu.latent(2, 12, 4, 10, 20, 6, 0.3, lu.dense(20))
    c = lu.conf([one, one], 24, 40, streams=1)
    W = oracle.random_weights(c, seed=6)
    eng = lu.make_engine(c, W, max_model_len=64, kv_block_size=8)
    seq = lu.tokens(30, 40, 1)
    lu.assert_close(lu.run_alone(eng, seq, [11, 1, 2]), oracle.forward(W, c, seq))
    a, b = eng.generate([seq[:9]], SamplingParams(max_new_tokens=8, greedy=True), n=2)
    assert a.out_tokens == b.out_tokens == _greedy(W, c, seq[:9], 8)


def test_greedy_generation_with_shared_prompts_and_stops():
    c = lu.uneven_conf()
    W = oracle.random_weights(c, seed=6)
    eng = lu.make_engine(c, W, max_model_len=48, kv_block_size=4, max_prefill_tokens=6, sync_interval=4)
    prompts = [lu.tokens(n, 75, 80 + n) for n in (1, 4, 9, 15)]
    want = [_greedy(W, c, p, 8) for p in prompts]
    for k, r in enumerate(eng.generate(prompts, SamplingParams(max_new_tokens=8, greedy=True), n=2)):
        assert r.out_tokens == want[k // 2] and r.finish_reason == "length"
    stop = want[0][3]
    for w, r in zip(want, eng.generate(prompts, SamplingParams(max_new_tokens=8, greedy=True, stop_token_ids=(stop,)))):
        assert r.out_tokens == (w[:w.index(stop) + 1] if stop in w else w)
    assert eng.get_load()["free_blocks"] == eng.num_blocks
    eng.sleep()
    assert not eng.k_cache
    assert eng.generate(prompts[:1], SamplingParams(max_new_tokens=8, greedy=True))[0].out_tokens == want[0]


def test_sampling_is_per_request_and_reproducible():
    c = lu.uneven_conf()
    eng = lu.make_engine(c, oracle.random_weights(c, seed=7), max_model_len=32)
    runs = [eng.generate([[5, 6, 7]], SamplingParams(max_new_tokens=6, seed=3, temperature=3.0), n=4) for _ in range(2)]
    assert [r.out_tokens for r in runs[0]] == [r.out_tokens for r in runs[1]]
    assert len({tuple(r.out_tokens) for r in runs[0]}) > 1


def test_gated_experts_without_normalisation():
    torch.manual_seed(1)
    T, E, K = 20, 12, 3
    counts = torch.zeros(E, dtype=torch.int32)
    logits, corr = torch.randn(T, E), torch.randn(E) * 0.2 - 2
    idx, w, _ = moe.choose(logits, E, K, corr, counts, sigmoid=True, norm=False, scale=2.0, groups=6, keep=2)
    router = dict(top=K, scale=2.0, groups=dict(count=6, keep=2))
    for t in range(T):
        ref = dict(oracle.choose_experts(logits[t].double(), corr.double(), router))
        assert set(idx[t].tolist()) == set(ref)
        assert all(abs(x - ref[e]) < 1e-6 for e, x in zip(idx[t].tolist(), w[t].tolist()))
    idx, _, _ = moe.choose(logits, E, 2, corr, counts, sigmoid=True, groups=12, keep=2)       # groups of one expert
    assert torch.equal(idx.sort(-1).values, (torch.sigmoid(logits) + corr).topk(2).indices.sort(-1).values)

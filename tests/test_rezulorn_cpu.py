"""Rezulorn on the CPU: configuration and layer plan, checkpoint reading, the engine's scheduling (portions, mixed batches,
freed pages and slots, generation) against whole sequences of the plain implementation, and that implementation itself."""
import copy
import json
import math

import pytest
import torch

from gcore_b200.models.config import MODEL_ARCH, from_hf_config
from gcore_b200.models.layer_plan import ConvLayerSpec, RetentionSpec, RotarySpec, ScoredAttentionSpec
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.ops import conv_norm as cn
from gcore_b200.rollout.engine import RolloutWeights, SamplingParams
from tests import rezulorn_util as ru
from tests.oracle import rezulorn as oracle


# ---------------------------------------------------------------------------------------------- configuration, loading
def test_config_is_read_layer_by_layer():
    c = ru.uneven_conf()
    cfg = from_hf_config(json.loads(json.dumps(c)))
    assert cfg.arch == "rezulorn" and cfg.arch in MODEL_ARCH and cfg.vocab_size == 75 and cfg.hidden_size == 44
    assert not cfg.tie_word_embeddings and cfg.rms_norm_eps == 1e-5 and cfg.num_layers == 7
    plan = cfg.layer_plan
    assert (plan.taps, plan.residual_mult, plan.logit_scale) == (4, 0.8, 1.5) and [r.layer for r in plan.runs] == list(range(7))
    a, p, g = plan.layers[0], plan.layers[1], plan.layers[2]
    m = a.mixers[0]
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.keep, m.scale) == (6, 2, 20, 12, 9, 3, 0.3)
    assert (m.weights, m.distance, m.head_bias, m.unit, m.rot) == ("softmax", True, False, False, None)
    left, right = p.mixers
    assert p.scales == (0.7, 1.3) and (left.weights, left.unit, left.head_bias, left.window) == ("sigmoid", True, True, 0)
    assert left.rot == RotarySpec(dims=6, base=90.0, slow=3.0, halves=True) and right.rot.slow == 1.0
    assert (right.norm, right.gate, right.act) == ("head", "silu", "") and right.product_scale() == pytest.approx(10 ** -0.5)
    r = g.mixers[0]
    assert (r.act, r.norm, r.gate, r.rot, r.product_scale(), r.decay) == ("silu", "joint", "sigmoid", None, 1.0, (0.999, 0.5, 0.9))
    assert a.ffn.act == "relu2" and g.ffn is None
    unread = [f"l{i}.{n}2" for i in (2, 3, 4) for n in ("norm", "canon")]
    assert cfg.num_parameters() == sum(t.numel() for k, t in oracle.random_weights(c).items() if k not in unread)


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Unknown"), lambda c: c["layers"][0].update(type="other"), lambda c: c.update(layers=[]),
    lambda c: c["layers"][0]["mixer"].pop("mask"), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"]["mask"].pop("keep_first"), lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"].pop("left_scale"), lambda c: c["layers"][1]["mixer"]["left"].pop("rot"),
    lambda c: c["layers"][1]["mixer"]["right"].pop("rot"), lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=14),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=5), lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(factor=0), lambda c: c["layers"][2]["mixer"].pop("vdim"),
    lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.5, 1.5]), lambda c: c["layers"][0]["mlp"].update(kind="other"),
    lambda c: c["layers"][0].update(mlp=dict(kind="moe", router=dict(experts=2, top=1), expert=dict(ff=4))),
    lambda c: c.pop("residual_mult"), lambda c: c.pop("logit_scale"), lambda c: c.pop("canon"), lambda c: c["canon"].update(taps=0)])
def test_what_the_design_does_not_have_is_refused(edit):
    c = copy.deepcopy(ru.uneven_conf())
    edit(c)
    with pytest.raises((ValueError, KeyError)):
        from_hf_config(c)


def test_specs_refuse_what_no_kernel_computes():
    with pytest.raises(ValueError):
        ScoredAttentionSpec(2, 1, 8, 8, 0.1, weights="linear")
    with pytest.raises(ValueError):
        RetentionSpec(1, 8, 8, (0.5,), norm="joint", gate="silu")
    with pytest.raises(ValueError):
        RetentionSpec(1, 8, 8, (0.5,), act="silu", rot=RotarySpec(4, 10.0))
    with pytest.raises(ValueError):
        ConvLayerSpec((), ())
    with pytest.raises(ValueError, match="taps"):
        build_decoder(from_hf_config(ru.uneven_conf(taps=17)))
    with pytest.raises(ValueError, match="width"):
        build_decoder(from_hf_config(ru.conf([ru.lightning(1, 8, 8, [0.5], None)], 17000, 4)))


def test_halves_become_neighbours():
    assert RotarySpec(6, 10.0, halves=True).neighbours(8) == [0, 3, 1, 4, 2, 5, 6, 7]
    assert RotarySpec(4, 10.0).neighbours(5) == [0, 1, 2, 3, 4]
    assert RotarySpec(4, 100.0, slow=4.0).frequencies() == pytest.approx([0.25, 0.025])


def test_checkpoint_tensors_must_fit_exactly():
    c = ru.uneven_conf()
    W = oracle.random_weights(c)
    cfg = from_hf_config(c)
    for bad in ({k: v for k, v in W.items() if k != "l0.mix.r2"}, {**W, "l0.mix.left.q": W["l0.mix.q"]},
                {**W, "l0.mix.o": W["l0.mix.o"][:, :-1]}, {**W, "l1.canon2": W["l1.canon2"][:, :-1]},
                {k: v for k, v in W.items() if k != "l1.mix.left.pb"}, {k: v for k, v in W.items() if k != "l6.mix.norm"}):
        with pytest.raises((KeyError, ValueError)):
            build_decoder(cfg).load_tensors(bad)
    m = build_decoder(cfg).load_tensors(W)
    sub = m.layers[1].mixer        # both mixers in one matrix; padded heads: real rows in place, zero rows between them
    left, right = sub.parts
    k = sub.in_proj[left.layout.k:left.layout.k + left.layout.dim]
    order = [0, 3, 1, 4, 2, 5, 6, 7, 8, 9, 10, 11]
    assert torch.equal(k[:12, :44], W["l1.mix.left.k"].float()[order]) and not k[12:].any() and not k[:, 44:].any()
    g = sub.in_proj[left.columns + right.at[3]:][:2 * right.vdim].view(2, right.vdim, -1)
    assert torch.equal(g[:, :20, :44], W["l1.mix.right.g"].float().view(2, 20, 44)) and not g[:, 20:].any()
    o = sub.out_proj[:44, left.out_columns:].view(44, 2, right.vdim)
    assert torch.equal(o[..., :20], W["l1.mix.right.o"].float().view(44, 2, 20)) and not o[..., 20:].any()
    assert torch.equal(sub.taps[-1, :44], W["l1.canon1"].float()[:, 3] + 1) and torch.equal(sub.taps[0, :44], W["l1.canon1"].float()[:, 0])
    drop = {k: v for k, v in W.items() if k not in ("l2.norm2", "l2.canon2")}     # no feed-forward: nothing reads them
    build_decoder(cfg).load_tensors(drop)


def test_layers_ask_for_the_cache_and_state_they_use():
    c = ru.uneven_conf()
    eng = ru.make_engine(c, oracle.random_weights(c), max_model_len=32)
    eng.wake_up()
    assert [x is None for x in eng.k_cache] == [False, False, True, False, False, False, True]
    assert [s.memory is None for s in eng.memory] == [True, False, False, True, False, True, False]
    assert [len(s.rings) for s in eng.memory] == [2, 2, 1, 1, 1, 2, 2] and eng.memory[0].rings[0].shape == (4, 3, 48)
    assert eng.k_cache[0].shape[2:] == (2 * 24 + 2 * 16,) and eng.memory[1].memory.S.shape == (4, 2, 16, 32)
    rows = sum(x[0, 0].numel() for x in eng.k_cache if x is not None)
    assert eng._kv_bytes_per_block() == rows * eng.bs * 4
    held = sum(t[0].numel() for s in eng.memory for t in s.rings + ([s.memory.S] if s.memory is not None else []))
    assert eng.plan.state_bytes_per_slot() == 4 * held


def test_registered_and_served_only():
    from gcore_b200 import build_native
    from gcore_b200.models.config import build_model_config
    from gcore_b200.models.gpt import GPTModel
    from gcore_b200.ops import registry
    c = ru.uneven_conf()
    assert build_model_config("rezulorn", {"hf_config": c}).layer_plan == from_hf_config(c).layer_plan
    with pytest.raises(ValueError, match="config.json"):
        build_model_config("rezulorn")
    with pytest.raises(ValueError, match="served"):
        GPTModel(from_hf_config(c))
    eng = ru.make_engine(c, oracle.random_weights(c), max_model_len=32)
    with pytest.raises(NotImplementedError):
        eng.quantize_weights_fp8()
    assert {"scored_attention", "retention", "conv_add_sublayer", "head_prep"} <= set(registry.available())
    assert all((build_native.OPS_SRC / f"{s}.cu").exists() for s in build_native.KERNEL_SETS["rezulorn"])


def test_new_weights_replace_the_old_ones():
    c = ru.uneven_conf()
    Wa, Wb = oracle.random_weights(c, seed=1), oracle.random_weights(c, seed=2)
    eng = ru.make_engine(c, Wa, max_model_len=64)
    seq = ru.tokens(20, 75, 1)
    eng.update_weights(RolloutWeights.from_model(build_decoder(eng.cfg).load_tensors(Wb)))
    ru.assert_close(ru.run_alone(eng, seq, [20]), ru.forward(Wb, c, seq))
    eng.load_weights_from(build_decoder(eng.cfg).load_tensors(Wa))
    ru.assert_close(ru.run_alone(eng, seq, [20]), ru.forward(Wa, c, seq))


# --------------------------------------------------------------------------------------------------------- plain oracle
def test_plain_rotation_turns_halves_and_keeps_distances():
    rot = ru.rotation(4, 50.0, 2.5)
    torch.manual_seed(0)
    q, k = torch.randn(1, 1, 6).double(), torch.randn(1, 1, 6).double()
    at = lambda x, p: oracle.rotate(x, rot, [p])[0, 0]
    assert float(at(q, 9) @ at(k, 4)) == pytest.approx(float(at(q, 905) @ at(k, 900)))    # only the distance counts
    assert torch.equal(at(q, 7)[4:], q[0, 0, 4:])
    one = torch.zeros(1, 1, 6).double()
    one[0, 0, 1] = 1.0                                                                    # second pair: dimensions 1 and 3
    y, a = at(one, 3), 3 * 50.0 ** (-2 / 4) / 2.5
    assert y[1] == pytest.approx(math.cos(a)) and y[3] == pytest.approx(math.sin(a)) and y[[0, 2, 4, 5]].abs().sum() == 0


def test_plain_window_with_kept_positions_by_hand():
    see = lambda i, size, keep: oracle.visible(i, dict(size=size, keep_first=keep))
    assert oracle.visible(4) == [0, 1, 2, 3, 4] and see(5, 1, 0) == [5] and see(5, 2, 1) == [0, 4, 5]
    assert see(6, 3, 2) == [0, 1, 4, 5, 6] and see(3, 3, 2) == [0, 1, 2, 3] and see(2, 2, 9) == [0, 1, 2]


def test_plain_scores_by_hand():
    d = torch.tensor([0.0, 3.0]).double()
    assert torch.allclose(oracle.distance_penalty(d, 2.0, 1.0), torch.tensor([0.0, 2 * math.log(4.0)]).double())
    k, v = torch.zeros(2, 1).double(), torch.tensor([[1.0], [5.0]]).double()
    got = oracle.softmax_attention(k, k, v, 1.0, dict(size=9, keep_first=0), 1.0, 1.0)    # weights 1/2 : 1
    assert float(got[1]) == pytest.approx((0.5 * 1 + 5) / 1.5)
    got = oracle.sigmoid_attention(k, k, v, 1.0, math.log(3.0))                           # each weight 3/4, not normalised
    assert float(got[1]) == pytest.approx(0.75 * 6)


def test_plain_memory_and_convolution_by_hand():
    q, k, v = (torch.tensor(x).double().view(3, 1) for x in ([1.0, 1.0, 2.0], [1.0, 2.0, 3.0], [1.0, 1.0, 10.0]))
    assert oracle.fading_memory(q, k, v, 0.5).flatten().tolist() == [1.0, 2.5, 2 * (1.25 + 30)]
    h = torch.tensor([[1.0], [10.0], [100.0]]).double()
    assert oracle.input_conv(h, torch.tensor([[3.0, 2.0]]).double()).flatten().tolist() == [3.0, 33.0, 330.0]
    y = oracle.layer_norm(torch.tensor([[1.0, 3.0]]).double(), torch.tensor([1.0, 2.0]).double(), 0.0)
    assert y.flatten().tolist() == [-1.0, 2.0]


FAULTS = ["window", "kept", "kept one less", "kept positions", "penalty", "r1", "r2", "log base", "scale", "gate scale", "pb", "softmax",
          "unit", "pairs", "dims", "scaling", "rotate values", "retention rotation", "key scale", "decay", "decay order", "head norm",
          "silu gate", "left scale", "right scale", "silu values", "silu keys", "joint norm", "joint gain", "sigmoid gate",
          "group", "conv", "conv order", "conv residual", "canon2", "centre", "eps", "relu2", "mult", "logits", "final norm"]


@pytest.mark.parametrize("fault", FAULTS)
def test_a_planted_mistake_shows(fault, monkeypatch):
    """The test models are sensitive: one wrong piece in the plain implementation moves the logits far beyond rounding."""
    c = ru.uneven_conf()
    W = oracle.random_weights(c, seed=2)
    seq = ru.tokens(60, 75, 3)
    eng = ru.make_engine(c, W, max_model_len=128)
    got = ru.run_alone(eng, seq, [60])
    ru.assert_close(got, ru.forward(W, c, seq))
    bad, Wb = json.loads(json.dumps(c)), dict(W)
    fill = lambda end, f: Wb.update({k: f(v) for k, v in W.items() if k.endswith(end)})
    mixers = lambda kind: [sp["mixer"] for sp in bad["layers"] if sp["type"] == kind]
    was = {n: getattr(oracle, n) for n in ("visible", "rotate", "fading_memory", "rms", "silu", "heads_of", "input_conv",
                                           "layer_norm", "distance_penalty")}
    plant = lambda name, f: monkeypatch.setattr(oracle, name, f)
    if fault == "window":
        for m in mixers("attention"):
            m["mask"]["size"] += 1
    elif fault == "kept":
        for m in mixers("attention"):
            m["mask"]["keep_first"] = 0
    elif fault == "kept one less":
        mixers("attention")[0]["mask"]["keep_first"] -= 1
    elif fault == "kept positions":       # distances of kept keys as if they lay just in front of the window
        plant("distance_penalty", lambda d, r1, r2: was["distance_penalty"](d.clamp_max(9.0), r1, r2))
    elif fault == "penalty":
        plant("distance_penalty", lambda d, r1, r2: 0 * d)
    elif fault == "r1":
        fill(".r1", lambda v: v.flip(0))
    elif fault == "r2":
        fill(".r2", lambda v: v.flip(0))
    elif fault == "log base":
        plant("distance_penalty", lambda d, r1, r2: r1 * torch.log2(1 + r2 * d))
    elif fault == "scale":
        for m in mixers("attention"):
            m["scale"] *= 1.1
    elif fault == "gate scale":
        for m in mixers("parallel"):
            m["left"]["scale"] *= 1.1
    elif fault == "pb":
        fill(".pb", lambda v: v.flip(0))
    elif fault == "softmax":
        plant("sigmoid_attention", lambda q, k, v, s, b: oracle.softmax_attention(q, k, v, s, None, 0.0, 0.0))
    elif fault == "unit":
        plant("rms", lambda x, eps: x if x.dim() == 3 else was["rms"](x, eps))
    elif fault == "pairs":                # neighbours in place of halves
        def neighbours(x, rot, p):
            n = rot["dims"]
            order = [i // 2 + (i % 2) * (n // 2) for i in range(n)] + list(range(n, x.shape[-1]))
            return was["rotate"](x[..., torch.tensor(order).argsort()], rot, p)[..., order]
        plant("rotate", neighbours)
    elif fault == "dims":
        bad["layers"][1]["mixer"]["left"]["rot"]["dims"] += 2
    elif fault == "scaling":
        bad["layers"][1]["mixer"]["left"]["rot"].pop("scaling")
    elif fault == "rotate values":
        plant("heads_of", lambda W, n, h, k: was["rotate"](was["heads_of"](W, n, h, k), ru.rotation(4, 20.0), range(h.shape[0]))
              if n.endswith("left.v") else was["heads_of"](W, n, h, k))
    elif fault == "retention rotation":
        for m in mixers("parallel"):
            m["right"]["rot"]["base"] *= 2
    elif fault == "key scale":            # only eps of the head norm sees it: tiny states
        bad["norm"]["eps"] = c["norm"]["eps"] = 0.3
        eng = ru.make_engine(c, W, max_model_len=128)
        got = ru.run_alone(eng, seq, [60])
        ru.assert_close(got, ru.forward(W, c, seq))
        plant("fading_memory", lambda q, k, v, d: was["fading_memory"](q, k * 2, v, d))
    elif fault == "decay":
        bad["layers"][1]["mixer"]["right"]["decay"][0] += 0.05
    elif fault == "decay order":
        bad["layers"][2]["mixer"]["decay"].reverse()
    elif fault == "head norm":
        plant("rms", lambda x, eps: x if x.dim() == 2 and x.shape[1] in (20, 6) else was["rms"](x, eps))
    elif fault == "silu gate":
        fill("right.g", lambda v: -v)
    elif fault == "left scale":
        for m in mixers("parallel"):
            m["left_scale"] = 1.0
    elif fault == "right scale":
        for m in mixers("parallel"):
            m["right_scale"] = 1.0
    elif fault in ("silu values", "silu keys"):
        count = [0]

        def silu(z):
            count[0] += z.dim() == 3
            return z if z.dim() == 3 and count[0] % 3 == (0 if fault == "silu values" else 2) else was["silu"](z)
        plant("silu", silu)
    elif fault == "joint norm":           # per head in place of all heads together
        plant("rms", lambda x, eps: was["rms"](x.view(-1, 3, 20), eps).view(-1, 60) if x.shape[-1] == 60 else was["rms"](x, eps))
    elif fault == "joint gain":
        fill("mix.norm", torch.ones_like)
    elif fault == "sigmoid gate":
        fill("l2.mix.g", lambda v: 0 * v)
    elif fault == "group":                # another key/value head
        fill("l0.mix.k", lambda v: v.view(2, 20, -1).flip(0).reshape(v.shape))
    elif fault == "conv":
        plant("input_conv", lambda h, w: h)
    elif fault == "conv order":
        fill("canon1", lambda v: v.flip(1))
    elif fault == "conv residual":
        plant("input_conv", lambda h, w: was["input_conv"](h, w) - h)
    elif fault == "canon2":
        Wb.update({k.replace("canon1", "canon2"): v for k, v in W.items() if k.endswith("canon1")})
    elif fault == "centre":
        plant("layer_norm", lambda x, w, eps: was["rms"](x, eps) * w)
    elif fault == "eps":
        bad["norm"]["eps"] = 1e-1
    elif fault == "relu2":
        plant("feed_forward", lambda W, p, h: torch.relu(h @ W[p + "up"].T) @ W[p + "down"].T)
    elif fault == "mult":
        bad["residual_mult"] = 1.0
    elif fault == "logits":
        bad["logit_scale"] = 1.0
    else:
        Wb["final.norm"] = torch.ones_like(W["final.norm"])
    assert ru.rms_error(got, ru.forward(Wb, bad, seq)).max() > 1e-2


# --------------------------------------------------------------------------------------------------------------- engine
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_portions_match_the_whole_prompt(taps):
    c = ru.uneven_conf(taps)
    W = oracle.random_weights(c, seed=4)
    eng = ru.make_engine(c, W, max_model_len=128, kv_block_size=8)
    for n in (1, 2, 39, 77):
        seq = ru.tokens(n, 75, n)
        want = ru.forward(W, c, seq)
        for cuts in ([n], [1], [2], [7, 1, 3], [36, 2, 1]):
            ru.assert_close(ru.run_alone(eng, seq, cuts), want, what=(n, cuts))
    st = eng.get_load()
    assert st["free_blocks"] == st["num_blocks"] and st["running"] == 0


def test_residual_after_every_layer():
    c = ru.uneven_conf()
    W = oracle.random_weights(c, seed=5)
    eng = ru.make_engine(c, W, max_model_len=64)
    eng.wake_up()
    seq, got = ru.tokens(17, 75, 9), []
    want = oracle.forward(W, c, seq)[1]
    rid = eng.open_request()
    assert eng.sched.reserve(rid, 17) == 0
    rows, _ = eng._step_rows([(rid, 0, seq)])
    eng.plan(rows, eng.k_cache, eng.memory, record=got)
    assert len(got) == len(want) == 7
    for g, w in zip(got, want):
        assert (g[:, :44] - w).abs().max() < 1e-4 * w.abs().max()


def test_mixed_requests_on_a_small_pool():
    """Nine requests through four slots and a pool that only holds four: pages and slots are used again."""
    c = ru.uneven_conf()
    W = oracle.random_weights(c, seed=5)
    eng = ru.make_engine(c, W, max_model_len=64, kv_block_size=4, num_kv_blocks=48)
    seqs = [ru.tokens(n, 75, 60 + n) for n in (40, 7, 21, 1, 44, 13, 30, 2, 39)]
    for s, got in zip(seqs, ru.run_mixed(eng, seqs, [1, 1, 2, 5, 9, 17], seed=1)):
        ru.assert_close(got, ru.forward(W, c, s))
    assert eng.get_load()["free_blocks"] == 48


@pytest.mark.parametrize("kind", ["attention", "lightning", "parallel"])
def test_plans_of_one_kind_of_layer(kind):
    one = dict(attention=ru.attention(4, 1, 12, 10, 6, 2, 0.3, 20), lightning=ru.lightning(2, 12, 10, [0.9, 0.99], 20),
               parallel=ru.parallel(ru.gates(2, 2, 8, 8, ru.rotation(8, 30.0), 0.4), ru.retention(1, 8, 4, ru.rotation(8, 30.0), [0.9]),
                                    1.0, 1.0, 20))[kind]
    c = ru.conf([one, one], 24, 40, taps=2, mult=1.0, logits=1.0)
    W = oracle.random_weights(c, seed=6)
    eng = ru.make_engine(c, W, max_model_len=64, kv_block_size=8)
    seq = ru.tokens(30, 40, 1)
    ru.assert_close(ru.run_alone(eng, seq, [11, 1, 2]), ru.forward(W, c, seq))
    a, b = eng.generate([seq[:9]], SamplingParams(max_new_tokens=8, greedy=True), n=2)
    assert a.out_tokens == b.out_tokens == oracle.greedy(W, c, seq[:9], 8)


def test_greedy_generation_with_shared_prompts_and_stops():
    c = ru.uneven_conf()
    W = oracle.random_weights(c, seed=6)
    eng = ru.make_engine(c, W, max_model_len=48, kv_block_size=4, max_prefill_tokens=6, sync_interval=4)
    prompts = [ru.tokens(n, 75, 80 + n) for n in (1, 4, 9, 15)]
    want = [oracle.greedy(W, c, p, 8) for p in prompts]
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
    c = ru.uneven_conf()
    eng = ru.make_engine(c, oracle.random_weights(c, seed=7), max_model_len=32)
    runs = [eng.generate([[5, 6, 7]], SamplingParams(max_new_tokens=6, seed=3, temperature=3.0), n=4) for _ in range(2)]
    assert [r.out_tokens for r in runs[0]] == [r.out_tokens for r in runs[1]]
    assert len({tuple(r.out_tokens) for r in runs[0]}) > 1


def test_a_convolution_reads_only_its_own_request():
    """Two requests and an inactive row in one batch: rings by slot, positions in front of the sequence are zero."""
    torch.manual_seed(0)
    rows = ru.make_rows([(0, 3), (5, 4), (2, 1), (7, 1)], 4, 16, 6, device="cpu")
    rows.states[3] = -1
    spec, n, H = cn.NormSpec(6, 1e-5), 4, 8
    taps, ring, h = torch.randn(n, H), torch.randn(6, n - 1, H), torch.randn(9, H)
    before = ring.clone()
    out = cn._convolve(h, taps, ring, rows)
    a, b, s = (int(rows.states[i]) for i in range(3))
    past = lambda slot, p: before[slot, p % 3] if p >= 0 else torch.zeros(H)
    assert torch.allclose(out[0], taps[3] * h[0]) and torch.allclose(out[2], taps[1] * h[0] + taps[2] * h[1] + taps[3] * h[2])
    assert torch.allclose(out[3], sum(taps[j] * past(b, 2 + j) for j in range(3)) + taps[3] * h[3])
    assert torch.allclose(out[7], taps[1] * past(s, 0) + taps[2] * past(s, 1) + taps[3] * h[7], atol=1e-6)
    assert torch.allclose(out[8], taps[3] * h[8])
    assert torch.equal(ring[a], h[:3]) and torch.equal(ring[b], h[[4, 5, 6]].roll(0, 0)[[(0 - 6) % 3, (1 - 6) % 3, (2 - 6) % 3]])
    assert torch.equal(ring[s, 2], h[7]) and torch.equal(ring[s, :2], before[s, :2])
    rest = [i for i in range(6) if i not in (a, b, s)]
    assert torch.equal(ring[rest], before[rest])
    d = cn.norm(h, torch.ones(H), spec)
    assert not d[:, 6:].any() and d[:, :6].mean(-1).abs().max() < 1e-6

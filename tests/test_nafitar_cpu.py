"""Nafitar on the CPU: configuration and layer plan, checkpoint reading, the engine's scheduling (portions, mixed batches,
freed pages and slots, generation) against whole sequences of the plain implementation, and that implementation itself."""
import copy
import json

import pytest
import torch

from gcore_b200.models.config import MODEL_ARCH, from_hf_config
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.rollout.engine import RolloutWeights, SamplingParams
from tests import nafitar_util as nu
from tests.oracle import nafitar as oracle


# ---------------------------------------------------------------------------------------------- configuration, loading
def test_config_is_read_layer_by_layer():
    c = nu.uneven_conf()
    cfg = from_hf_config(json.loads(json.dumps(c)))
    assert cfg.arch == "nafitar" and cfg.arch in MODEL_ARCH and cfg.vocab_size == 75 and cfg.hidden_size == 44
    plan = cfg.layer_plan
    assert [(s.attention.window, s.memory.vdim, s.ffn) for s in plan.layers] == [(37, 20, 36), (5, 24, 0), (2, 70, 44)]
    assert [(r.layer, r.opens_pass) for r in plan.runs] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None)]
    assert [r.index for r in plan.runs] == list(range(7))
    assert plan.layers[0].attention.slopes() == oracle.slopes(6)
    W = oracle.random_weights(c)
    assert cfg.num_parameters() == sum(t.numel() for t in W.values())
    del c["loop"]
    assert [(r.layer, r.opens_pass) for r in from_hf_config(c).layer_plan.runs] == [(0, None), (1, None), (2, None)]


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Unknown"), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=8), lambda c: c["layers"][0]["mlp"].update(kind="other"),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), lambda c: c["loop"].update(stop=9),
    lambda c: c["layers"][2]["mixer"]["left"]["mask"].update(size=0)])
def test_what_the_design_does_not_have_is_refused(edit):
    c = copy.deepcopy(nu.uneven_conf())
    edit(c)
    with pytest.raises((ValueError, KeyError)):
        from_hf_config(c)


def test_checkpoint_tensors_must_fit_exactly():
    c = nu.uneven_conf(positions=32)
    W = oracle.random_weights(c)
    cfg = from_hf_config(c)
    for bad in ({k: v for k, v in W.items() if k != "l1.mix.right.i.b"}, {**W, "l1.norm2": W["l0.norm2"]},
                {**W, "l0.mix.left.o": W["l0.mix.left.o"][:, :-1]}):
        with pytest.raises((KeyError, ValueError)):
            build_decoder(cfg).load_tensors(bad)
    m = build_decoder(cfg).load_tensors(W)
    ly = m.layers[0]   # padded heads: real rows in place, zero rows between them
    q = ly.in_proj[ly.off["q"]:ly.off["k"]].view(6, ly.att_dim, -1)
    assert torch.equal(q[:, :20, :44].reshape(120, 44), W["l0.mix.left.q"]) and not q[:, 20:].any() and not q[..., 44:].any()


def test_serving_copy_owns_its_weights():
    c = nu.uneven_conf(positions=32)
    m = build_decoder(from_hf_config(c)).load_tensors(oracle.random_weights(c))
    shared, own = RolloutWeights.from_model(m), RolloutWeights.from_model(m, clone=True)
    assert shared.plan is m and own.plan is not m
    assert all(a.data_ptr() != b.data_ptr() and torch.equal(a, b) for a, b in zip(shared.tensors(), own.tensors()))


def test_registered_and_served_only():
    from gcore_b200 import build_native
    from gcore_b200.models.config import build_model_config
    from gcore_b200.models.gpt import GPTModel
    from gcore_b200.ops import registry
    c = nu.uneven_conf(positions=32)
    assert build_model_config("nafitar", {"hf_config": c}).layer_plan == from_hf_config(c).layer_plan
    with pytest.raises(ValueError, match="config.json"):
        build_model_config("nafitar")
    with pytest.raises(ValueError, match="served"):
        GPTModel(from_hf_config(c))
    eng = nu.make_engine(c, oracle.random_weights(c), max_model_len=32)
    with pytest.raises(NotImplementedError):
        eng.quantize_weights_fp8()
    assert {"window_attention", "matrix_memory", "add_sublayer"} <= set(registry.available())
    assert all((build_native.OPS_SRC / f"{s}.cu").exists() for s in build_native.KERNEL_SETS["nafitar"])


def test_new_weights_replace_the_old_ones():
    c = nu.uneven_conf(positions=64)
    Wa, Wb = oracle.random_weights(c, seed=1), oracle.random_weights(c, seed=2)
    eng = nu.make_engine(c, Wa, max_model_len=64)
    other = build_decoder(eng.cfg).load_tensors(Wb)
    seq = nu.tokens(20, 75, 1)
    eng.update_weights(RolloutWeights.from_model(other))
    nu.assert_close(nu.run_alone(eng, seq, [20]), oracle.forward(Wb, c, seq))
    eng.load_weights_from(build_decoder(eng.cfg).load_tensors(Wa))
    nu.assert_close(nu.run_alone(eng, seq, [20]), oracle.forward(Wa, c, seq))


# --------------------------------------------------------------------------------------------------------- plain oracle
def test_plain_window_and_distance_penalty_by_hand():
    """One head, keys that are all alike except one: the window keeps exactly ``size`` tokens."""
    m = dict(heads=1, kv_heads=1, dim=2, scale=1.0, mask=dict(size=4))
    W = {"a.q": torch.zeros(2, 2).double(), "a.q.b": torch.zeros(2).double(), "a.k": torch.eye(2).double(),
         "a.k.b": torch.zeros(2).double(), "a.o": torch.eye(2).double()}
    h = torch.zeros(9, 2).double()
    h[2, 0] = 1.0
    y = oracle.window_attention(W, "a", m, h)[:, 0]
    slope = 2.0 ** -8
    for t in range(9):
        lo = max(0, t - 3)
        p = torch.softmax(-slope * torch.arange(t - lo, -1, -1).double(), 0)
        assert abs(y[t] - (p[2 - lo] if lo <= 2 <= t else 0.0)) < 1e-12
    assert y[5] > 0 and y[6] == 0


def test_plain_memory_matches_its_sum_form():
    """The recurrence with its running maximum = the plain double sum, with and without a carried state."""
    torch.manual_seed(0)
    m = dict(heads=2, dim=3, vdim=5, gate_cap=4.0)
    W = {f"x.{k}": torch.randn(n, 6).double() for k, n in (("q", 6), ("k", 6), ("v", 10), ("i", 2), ("f", 2))}
    W["x.i.b"], W["x.f.b"] = torch.randn(2).double(), torch.randn(2).double()
    h = torch.randn(11, 6).double()
    whole = oracle.matrix_memory(W, "x", m, h, 1e-6, core=True)
    st = oracle.fresh_memory(m)
    parts = torch.cat([oracle.matrix_memory(W, "x", m, h[a:b], 1e-6, st, core=True) for a, b in ((0, 4), (4, 5), (5, 11))])
    assert (whole - parts).abs().max() < 1e-12
    f = torch.nn.functional.logsigmoid(4 * torch.tanh((h @ W["x.f"].T + W["x.f.b"]) / 4))
    i = 4 * torch.tanh((h @ W["x.i"].T + W["x.i.b"]) / 4)
    q, k, v = (h @ W["x.q"].T).view(-1, 2, 3) * 3 ** -0.5, (h @ W["x.k"].T).view(-1, 2, 3), (h @ W["x.v"].T).view(-1, 2, 5)
    for t in range(11):
        for a in range(2):
            w = torch.stack([torch.exp(i[s, a] + f[s + 1:t + 1, a].sum()) * (q[t, a] @ k[s, a]) for s in range(t + 1)])
            # m starts at zero: the floor of the denominator is e^-m, i.e. at least the weight of an empty start
            want = (w[:, None] * v[:t + 1, a]).sum(0)
            big = max([f[:t + 1, a].sum()] + [i[s, a] + f[s + 1:t + 1, a].sum() for s in range(t + 1)])
            den = max(abs(w.sum()) * torch.exp(-big), torch.exp(-big)) + 1e-6
            assert (whole[t, a] - want * torch.exp(-big) / den).abs().max() < 1e-10


@pytest.mark.parametrize("fault", ["window", "slope", "step", "first", "post", "eps"])
def test_a_planted_mistake_shows(fault, monkeypatch):
    """The test models are sensitive: one wrong constant in the plain implementation moves the logits far beyond rounding."""
    c = nu.uneven_conf(positions=128)
    W = oracle.random_weights(c, seed=2)
    seq = nu.tokens(60, 75, 3)
    eng = nu.make_engine(c, W, max_model_len=128)
    got = nu.run_alone(eng, seq, [60])
    nu.assert_close(got, oracle.forward(W, c, seq))
    bad, Wb = copy.deepcopy(c), dict(W)
    if fault == "window":
        bad["layers"][1]["mixer"]["left"]["mask"]["size"] += 1
    elif fault == "slope":
        right = oracle.slopes
        monkeypatch.setattr(oracle, "slopes", lambda n: [s / 2 for s in right(n)])
    elif fault == "step":
        Wb["loop.step"] = W["loop.step"].roll(1, 0)
    elif fault == "first":
        order = oracle.run_order(c)
        monkeypatch.setattr(oracle, "run_order", lambda _: [(i, t, o and t == 0) for i, t, o in order])
    elif fault == "post":
        Wb["l2.norm1b"] = torch.zeros_like(W["l2.norm1b"])
    else:
        bad["norm"]["eps"] = 1e-1
    assert nu.rms_error(got, oracle.forward(Wb, bad, seq)).max() > 1e-2


# --------------------------------------------------------------------------------------------------------------- engine
def test_portions_match_the_whole_prompt():
    c = nu.uneven_conf(positions=128)
    W = oracle.random_weights(c, seed=4)
    eng = nu.make_engine(c, W, max_model_len=128, kv_block_size=8)
    for n in (1, 2, 39, 77):
        seq = nu.tokens(n, 75, n)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [7, 1, 3], [36, 2, 1]):
            nu.assert_close(nu.run_alone(eng, seq, cuts), want, what=(n, cuts))
    st = eng.get_load()
    assert st["free_blocks"] == st["num_blocks"] and st["running"] == 0


def test_mixed_requests_on_a_small_pool():
    """Nine requests through four slots and a pool that only holds four: pages and slots are used again."""
    c = nu.uneven_conf(positions=64)
    W = oracle.random_weights(c, seed=5)
    eng = nu.make_engine(c, W, max_model_len=64, kv_block_size=4, num_kv_blocks=48)
    seqs = [nu.tokens(n, 75, 60 + n) for n in (40, 7, 21, 1, 44, 13, 30, 2, 39)]
    for s, got in zip(seqs, nu.run_mixed(eng, seqs, [1, 1, 2, 5, 9, 17], seed=1)):
        nu.assert_close(got, oracle.forward(W, c, s))
    assert eng.get_load()["free_blocks"] == 48


def test_step_refuses_what_does_not_fit():
    c = nu.uneven_conf(positions=32)
    eng = nu.make_engine(c, oracle.random_weights(c), max_model_len=32, kv_block_size=4, num_kv_blocks=9,
                         max_running_requests=2)
    a, b = eng.open_request(), eng.open_request()
    with pytest.raises(RuntimeError, match="slot"):
        eng.open_request()
    for bad in ([(a, [75])], [(a, [])], [(a, [1] * 33)], [(a, [1]), (a, [2])]):
        with pytest.raises(ValueError):
            eng.step(bad)
    with pytest.raises(ValueError):
        eng.step([(a, [1, 2])], [[2]])
    assert eng.step([(a, [1] * 30)]) is None
    with pytest.raises(RuntimeError, match="exhausted"):
        eng.step([(b, [1] * 8)])
    eng.close_request(a)
    assert eng.step([(b, [1] * 8)], [[7]]).shape == (1, 75)
    with pytest.raises(ValueError, match="positions"):
        nu.make_engine(c, oracle.random_weights(c), max_model_len=33)
    with pytest.raises(ValueError, match="max_model_len"):
        eng.generate([[1] * 20], SamplingParams(max_new_tokens=13))


def _greedy(W, c, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(oracle.forward(W, c, t)[-1].argmax()))
    return t[len(prompt):]


def test_greedy_generation_with_shared_prompts_and_stops():
    c = nu.uneven_conf(positions=64)
    W = oracle.random_weights(c, seed=6)
    eng = nu.make_engine(c, W, max_model_len=48, kv_block_size=4, max_prefill_tokens=6, sync_interval=4)
    prompts = [nu.tokens(n, 75, 80 + n) for n in (1, 4, 9, 15, 23)]
    want = [_greedy(W, c, p, 10) for p in prompts]
    for k, r in enumerate(eng.generate(prompts, SamplingParams(max_new_tokens=10, greedy=True), n=2)):
        assert r.out_tokens == want[k // 2] and r.finish_reason == "length"
    stop = want[0][3]
    for w, r in zip(want, eng.generate(prompts, SamplingParams(max_new_tokens=10, greedy=True, stop_token_ids=(stop,)))):
        assert r.out_tokens == (w[:w.index(stop) + 1] if stop in w else w)
    assert eng.get_load()["free_blocks"] == eng.num_blocks
    eng.sleep()
    assert not eng.memory and not eng.k_cache
    assert eng.generate(prompts[:1], SamplingParams(max_new_tokens=10, greedy=True))[0].out_tokens == want[0]


def test_sampling_is_per_request_and_reproducible():
    c = nu.uneven_conf(positions=64)
    eng = nu.make_engine(c, oracle.random_weights(c, seed=7), max_model_len=32)
    runs = [eng.generate([[5, 6, 7]], SamplingParams(max_new_tokens=6, seed=3, top_k=20), n=4) for _ in range(2)]
    assert [r.out_tokens for r in runs[0]] == [r.out_tokens for r in runs[1]]
    assert len({tuple(r.out_tokens) for r in runs[0]}) > 1

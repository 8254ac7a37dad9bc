"""Nafitar on the GPU: every kernel alone against the plain implementation, then the engine - portions, mixed batches,
freed pages and slots, long decoding, generation - against whole sequences of the plain implementation."""
import json

import pytest
import torch

from gcore_b200.ops import matrix_memory as mm
from gcore_b200.ops import sandwich
from gcore_b200.ops import window_attention as wa
from gcore_b200.rollout.engine import SamplingParams
from tests import nafitar_util as nu
from tests.oracle import nafitar as oracle

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


# ---------------------------------------------------------------------------------------------------- attention alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,window,bs", [(8, 2, 64, 70, 16), (6, 1, 128, 129, 64), (4, 4, 128, 1, 32), (20, 1, 64, 300, 8),
                                             (4, 2, 136, 33, 16), (4, 2, 64, 9, 12), (16, 1, 128, 1000, 128)])
def test_window_attention_alone(H, G, D, window, bs, dtype):
    """Random keys, and one query per request that singles out one key: the oldest visible one or the one just outside."""
    torch.manual_seed(1)
    segs = [(0, 150), (333, 70), (63, 2), (127, 65), (5, 2), (500, 1), (0, 1), (64, 1), (window + 3, 1), (255, 1)]
    total = [f + l for f, l in segs]
    rows = nu.make_rows(segs, bs, sum((t + bs - 1) // bs for t in total) + 5, 16)
    dt = DT[dtype]
    ld, q_off, k_off = H * D + G * D + 24, 8, 8 + H * D
    keys = [torch.randn(t, G, D).to(dt).double() for t in total]
    qs = [torch.randn(l, H, D).to(dt).double() for _, l in segs]
    scale = 0.11
    for (f, l), k, q in zip(segs, keys, qs):      # last row: heads alternate between the window's last key and the next one
        i = f + l - 1
        for h in range(H):
            j = i - window + (h % 2 == 0)
            if j >= 0:
                q[-1, h] = (k[j, h // (H // G)] * 6).to(dt).double()
    cache = torch.full((rows.tables.max().item() + 6, bs, G, D), 3.0, dtype=dt, device="cuda")
    flat = cache.view(-1, G, D)
    proj = torch.zeros(sum(l for _, l in segs), ld, dtype=dt, device="cuda")
    at = 0
    for s, (f, l) in enumerate(segs):
        p = torch.arange(f)
        flat[(rows.tables[s].cpu()[p // bs].long() * bs + p % bs).cuda()] = keys[s][:f].to(dt).cuda()
        proj[at:at + l, q_off:q_off + H * D] = qs[s].reshape(l, -1).to(dt).cuda()
        proj[at:at + l, k_off:k_off + G * D] = keys[s][f:].reshape(l, -1).to(dt).cuda()
        at += l
    sl = oracle.slopes(H)
    got = wa.window_attention(proj, q_off, k_off, H, G, D, rows, cache, torch.tensor(sl, device="cuda"), scale, window)
    got = got.view(-1, H, D).double().cpu()
    at = 0
    for s, (f, l) in enumerate(segs):
        for r in range(l):
            i = f + r
            lo = max(0, i - window + 1)
            for h in range(0, H, max(1, H // 5)):
                k = keys[s][lo:i + 1, h // (H // G)]
                sc = k @ qs[s][r, h] * scale - sl[h] * torch.arange(i - lo, -1, -1).double()
                want = torch.softmax(sc, 0) @ k
                err = (got[at + r, h] - want).abs().max() / want.abs().max().clamp_min(1.0)
                assert err < (2e-5 if dtype == "float32" else 8e-3), (s, r, h, float(err))
        p = torch.arange(f, f + l)                # the new keys went to their slots
        stored = flat[(rows.tables[s].cpu()[p // bs].long() * bs + p % bs).cuda()]
        assert torch.equal(stored.cpu().double(), keys[s][f:])
        at += l


def test_decode_splits_of_a_long_window_agree():
    """One request whose window is cut into many splits = the same with one split."""
    torch.manual_seed(2)
    H, G, D, window, bs = 8, 1, 128, 4000, 64
    rows = nu.make_rows([(5000, 1)], bs, 90, 2)
    cache = torch.randn(91, bs, G, D, device="cuda").bfloat16()
    proj = torch.randn(1, (H + G) * D, device="cuda").bfloat16()
    sl = torch.tensor(oracle.slopes(H), device="cuda")
    outs = []
    for target in (444, 1):
        wa._lib.kernels().gk_shared_decode_set_target_ctas(target)
        outs.append(wa.window_attention(proj, 0, H * D, H, G, D, rows, cache.clone(), sl, 0.09, window).float())
    wa._lib.kernels().gk_shared_decode_set_target_ctas(0)
    assert (outs[0] - outs[1]).abs().max() < 1e-2


# ------------------------------------------------------------------------------------------------- matrix memory alone
@pytest.mark.parametrize("finish", [0, 1 << 30])     # single tokens: output kernel behind the scan / finished in one launch
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim,width", [(3, 16, 16, 40), (2, 64, 128, 64), (2, 128, 80, 128), (1, 256, 64, 72),
                                                  (2, 144, 208, 64), (1, 320, 32, 48), (1, 32, 528, 40)])
def test_matrix_memory_alone(heads, dim, vdim, width, dtype, finish, monkeypatch):
    """Portions and single tokens with gates from nearly closed to wide open, carried state and fresh slots."""
    torch.manual_seed(3)
    dt = DT[dtype]
    segs = [(0, 300), (70, 130), (0, 2), (40, 7), (128, 128), (0, 1), (9, 1), (200, 1)]
    rows = nu.make_rows(segs, 16, 200, 12)
    ofs = [0, heads * dim, 2 * heads * dim, 2 * heads * dim + heads * vdim]
    ld = ofs[3] + heads * vdim
    m = dict(heads=heads, dim=dim, vdim=vdim, gate_cap=7.0)
    state = mm.MemoryState.allocate(12, heads, dim, vdim, "cuda")
    for t in (state.S, state.n, state.m):
        t.fill_(99.0)                                    # what earlier requests left
    gate_w = (torch.randn(2 * heads, width) * 0.6).to(dt)
    gate_b = torch.cat([torch.randn(heads), torch.randn(heads) * 3 + 1])
    q_scale = dim ** -0.5
    proj, hs, wants, states = [], [], [], []
    for s, (f, l) in enumerate(segs):
        pr, h = torch.randn(l, ld).to(dt), torch.randn(l, width).to(dt)
        gates = h.double() @ gate_w.double().T + gate_b.double()
        st = oracle.fresh_memory(m)
        if f:
            slot = int(rows.states[s])
            st = [(torch.randn(dim, vdim).double(), torch.randn(dim).double(), torch.randn(()).double()) for _ in range(heads)]
            for a, (S, n, mx) in enumerate(st):
                state.S[slot, a], state.n[slot, a], state.m[slot, a] = S.cuda(), n.cuda(), mx.cuda()
        # the plain implementation on ready projections: identity weights pick the blocks out of one wide input
        blocks = torch.cat([pr.double(), gates - gate_b.double()], 1)
        pick = lambda lo, n: torch.eye(blocks.shape[1], dtype=torch.float64)[lo:lo + n]
        W = {"x.q": pick(ofs[0], heads * dim), "x.k": pick(ofs[1], heads * dim), "x.v": pick(ofs[2], heads * vdim),
             "x.i": pick(ld, heads), "x.f": pick(ld + heads, heads), "x.i.b": gate_b[:heads].double(),
             "x.f.b": gate_b[heads:].double()}
        wants.append(oracle.matrix_memory(W, "x", m, blocks, 1e-5, st, core=True))
        states.append(st)
        proj.append(pr)
        hs.append(h)
    gain = torch.ones(heads * vdim, device="cuda")
    monkeypatch.setattr(mm, "FINISH_CTAS", finish)
    raw, output = [], mm._output
    monkeypatch.setattr(mm, "_output", lambda o, *a: raw.append(o.clone()) or output(o, *a))
    y = mm.matrix_memory(torch.cat(proj).cuda(), *ofs, torch.cat(hs).cuda(), gate_w.cuda(), gate_b.cuda(), 7.0, q_scale,
                         heads, dim, vdim, vdim, rows, state, gain, 1e-5)
    o, at = torch.cat(raw).double().cpu(), 0     # single tokens whose output is finished in one launch are not in it
    # bf16 inputs are exact in both: what is left is the two-term operands.  A few rows divide by a sum that nearly
    # cancels, hence the loose bound on the worst one beside the tight one on the mean.
    tol = 5e-4 if dtype == "float32" else 5e-3
    for s, (f, l) in enumerate(segs):
        if at < o.shape[0]:
            d = (o[at:at + l] - wants[s]).abs().amax(-1) / wants[s].abs().amax(-1).clamp_min(0.05)
            assert d.max() < tol and d.mean() < tol / 25, (s, float(d.max()), float(d.mean()), int(d.amax(-1).argmax()))
        slot = int(rows.states[s])
        for a, (S, n, mx) in enumerate(states[s]):
            assert (state.S[slot, a].cpu() - S).abs().max() < tol * S.abs().max().clamp_min(1e-2)
            assert (state.n[slot, a].cpu() - n).abs().max() < tol * n.abs().max().clamp_min(1e-2)
            assert (state.m[slot, a].cpu() - mx).abs().max() < 1e-4
        at += l
    g = torch.cat(proj)[:, ofs[3]:].double()
    want = oracle.rms(torch.cat(wants), 1e-5).reshape(at, -1) * torch.sigmoid(g)
    assert (y.double().cpu() - want).abs().max() < (2e-3 if dtype == "float32" else 6e-2)


# ---------------------------------------------------------------------------------------------------- residual kernels
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,pad", [(44, 48), (192, 192), (1000, 1000), (2048, 2048), (5000, 5000), (9000, 9000)])
def test_residual_steps_alone(width, pad, dtype):
    torch.manual_seed(4)
    dt, T, eps = DT[dtype], 5, 1e-3
    z = lambda t: torch.nn.functional.pad(t, (0, pad - width))
    x, y, y2 = torch.randn(T, width), torch.randn(T, width).to(dt), (torch.randn(T, width) * 3).to(dt)
    gains = [torch.rand(width) + 0.5 for _ in range(4)]
    first, step = torch.randn(T, width), torch.randn(width)
    c = lambda t: z(t).contiguous().cuda()
    for pair in (False, True):
        for extra in (False, True):
            xg = c(x)
            kw = dict(y2=c(y2), gain_a=c(gains[2]), gain_b=c(gains[3])) if pair else {}
            h = sandwich.add_sublayer(xg, c(y), c(gains[0]), width, eps, c(gains[1]), c(first) if extra else None,
                                      c(step) if extra else None, **kw)
            m = y.double()
            if pair:
                m = 0.5 * (oracle.rms(m, eps) * gains[2] + oracle.rms(y2.double(), eps) * gains[3])
            want = x.double() + oracle.rms(m, eps) * gains[0] + (first + step if extra else 0)
            assert (xg[:, :width].cpu() - want).abs().max() < 1e-5 and not xg[:, width:].any()
            assert (h[:, :width].cpu().double() - oracle.rms(want, eps) * gains[1]).abs().max() < \
                (2e-5 if dtype == "float32" else 3e-2)
    emb, pos = torch.randn(30, width).to(dt), torch.randn(20, width).to(dt)
    tok, ps = torch.tensor([3, 29, 0, 7, 7]), torch.tensor([0, 19, 5, 1, 2], dtype=torch.int32)
    xg, fg, h = sandwich.embed_rows(tok.cuda(), ps.cuda(), c(emb), c(pos), c(gains[0]), width, eps, c(step), keep_first=True)
    want = emb[tok].double() + pos[ps.long()].double()
    assert (fg[:, :width].cpu() - want).abs().max() < 1e-6 and (xg[:, :width].cpu() - want - step).abs().max() < 1e-5
    got = sandwich.norm_rows(xg, c(gains[1]), width, eps, dt, torch.tensor([4, 1], device="cuda"))
    want = oracle.rms((want + step)[[4, 1]], eps) * gains[1]
    assert (got[:, :width].cpu().double() - want).abs().max() < (2e-5 if dtype == "float32" else 3e-2)


# ---------------------------------------------------------------------------------------------------- engine
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["uneven", "round"])
def test_portions_and_decoding_match_whole_sequences(which, dtype):
    c = nu.uneven_conf() if which == "uneven" else nu.round_conf()
    W = oracle.random_weights(c, seed=5)
    eng = nu.make_engine(c, W, dtype, "cuda")
    for n, seed in ((1, 1), (2, 2), (150, 3), (333, 4)):
        seq = nu.tokens(n, c["vocab"], seed)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [64, 1], [15, 17, 1, 1, 100, 2]):
            if cuts == [1] and n > 200 or cuts == [2] and n < 200:
                continue
            nu.assert_close(nu.run_alone(eng, seq, cuts), want, dtype, (n, cuts))
    assert eng.get_load()["free_blocks"] == eng.num_blocks


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("block", [8, 64])
def test_mixed_batches_on_reused_pages_and_slots(dtype, block):
    c = nu.round_conf(window=33, loop=(1, 2, 3))
    W = oracle.random_weights(c, seed=6)
    eng = nu.make_engine(c, W, dtype, "cuda", kv_block_size=block, num_kv_blocks=4 * 256 // block, max_model_len=256)
    seqs = [nu.tokens(n, c["vocab"], 20 + n) for n in (200, 31, 64, 1, 129, 65, 90, 17, 240)]
    for s, got in zip(seqs, nu.run_mixed(eng, seqs, [1, 1, 2, 3, 16, 63, 64, 65, 100], seed=7)):
        nu.assert_close(got, oracle.forward(W, c, s), dtype)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_true_32_bit_whatever_the_matrix_mode():
    """The 32-bit engine stays exact when the process allows TF32."""
    c = nu.round_conf()
    W = oracle.random_weights(c, seed=8)
    eng = nu.make_engine(c, W, "float32", "cuda")
    seq = nu.tokens(70, c["vocab"], 9)
    torch.backends.cuda.matmul.allow_tf32 = True
    try:
        got = nu.run_alone(eng, seq, [40, 1])
    finally:
        torch.backends.cuda.matmul.allow_tf32 = False
    nu.assert_close(got, oracle.forward(W, c, seq))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype):
    """generate(): captured decode graphs, more requests than slots, prompts longer than a prefill step, samples that
    share a prompt - every token is the plain implementation's choice (or ties with it within rounding)."""
    c = nu.uneven_conf() if dtype == "float32" else nu.round_conf()
    W = oracle.random_weights(c, seed=10)
    eng = nu.make_engine(c, W, dtype, "cuda", max_prefill_tokens=50, sync_interval=3, max_model_len=256)
    prompts = [nu.tokens(n, c["vocab"], 40 + n) for n in (1, 5, 33, 120, 64)]
    reqs = eng.generate(prompts, SamplingParams(max_new_tokens=40, greedy=True), n=2)
    assert eng.stats["graph_replays"] > 0
    for k, r in enumerate(reqs):
        assert len(r.out_tokens) == 40 and r.out_tokens == reqs[k // 2 * 2].out_tokens
        if k % 2 == 0:
            lg = oracle.forward(W, c, r.prompt + r.out_tokens)[len(r.prompt) - 1:-1]
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert gap.max() < (1e-4 if dtype == "float32" else 0.25) * lg.std(), float(gap.max())
            lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert (lp - torch.tensor(r.out_logprobs)).abs().max() < (1e-3 if dtype == "float32" else 0.5)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_long_decoding_keeps_the_state():
    c = nu.conf([nu.layer_conf(4, 2, 64, 20, 0.15, 2, 32, 64, 6.0, 64)], width=64, vocab=128, positions=1024)
    W = oracle.random_weights(c, seed=11)
    eng = nu.make_engine(c, W, "bfloat16", "cuda", max_model_len=1024)
    seq = nu.tokens(600, c["vocab"], 12)
    got, want = nu.run_alone(eng, seq, [20] + [1] * 580), oracle.forward(W, c, seq)
    nu.assert_close(got, want, "bfloat16")


def test_command_line_generates_from_a_checkpoint_folder(tmp_path):
    from safetensors.torch import save_file

    from gcore_b200.entry import lm_infer
    c = nu.round_conf()
    W = oracle.random_weights(c, seed=13)
    save_file({k: v.contiguous() for k, v in W.items()}, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(c))
    prompts = [nu.tokens(n, c["vocab"], n) for n in (7, 20)]
    (tmp_path / "p.jsonl").write_text("".join(json.dumps({"prompt_token_ids": p}) + "\n" for p in prompts))
    out = tmp_path / "o.jsonl"
    lm_infer.main([f"checkpoint.load_ckpt_path={tmp_path}", f"+task.infer.prompts={tmp_path}/p.jsonl",
                   f"+task.infer.out={out}", "+task.infer.greedy=true"])
    eng = nu.make_engine(c, W, "bfloat16", "cuda", max_model_len=256)
    ref = eng.generate(prompts, SamplingParams(max_new_tokens=128, greedy=True))
    got = [json.loads(l) for l in out.read_text().splitlines()]
    assert [g["prompt_length"] for g in got] == [7, 20]
    for g, r in zip(got, ref):
        assert len(g["tokens"]) == g["prompt_length"] + 128 and g["tokens"][:40] == (r.prompt + r.out_tokens)[:40]


def test_trace_replay_through_the_executable_entry(tmp_path):
    import numpy as np

    from gcore_b200.entry import trace_run
    from safetensors.torch import save_file
    c = nu.uneven_conf()
    W = oracle.random_weights(c, seed=14)
    save_file({k: v.contiguous() for k, v in W.items()}, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(c))
    eng = trace_run.build_engine(str(tmp_path), "float32", 128, torch.device("cuda", 0))
    a, b = nu.tokens(40, c["vocab"], 1), nu.tokens(9, c["vocab"], 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[1:], want=[])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=b, want=[8]), dict(id="a", tokens=a[30:], want=[9])], end=["a", "c"])]
    said = []
    trace_run.replay(eng, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    la, lb = oracle.forward(W, c, a), oracle.forward(W, c, b)
    for n, want in ((0, torch.stack([la[0], la[29], lb[0]])), (2, torch.stack([lb[8], la[39]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"]).copy())
        nu.assert_close(got, want)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_serving_benchmark_runs_on_a_small_size():
    from gcore_b200.tools import serve_bench as sb
    s = dict(width=256, heads=4, kv=2, dim=128, window=100, mh=2, mk=64, mv=128, ff=512, layers=2)
    for kind in ("nafitar", "dense"):
        eng = sb.build(kind, s, 512, 4)
        assert sb.prefill_step(eng, 2, 130, 2) > 0 and sb.decode_step(eng, 4, 200, 2) > 0
    table = sb.kernel_table(s, 2, 130, 4, 200)
    assert {r[0] for r in table} == {"prefill", "decode"} and all(r[2] > 0 for r in table)

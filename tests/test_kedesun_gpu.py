"""Kedesun on the GPU: every kernel alone against the plain implementation, then the engine - portions, mixed batches,
freed pages and slots, long decoding, generation - against whole sequences of the plain implementation."""
import json

import pytest
import torch

from gcore_b200.models.config import from_hf_config
from gcore_b200.models.parallel_decoder import LatentAttentionMixer
from gcore_b200.models.plan_decoder import CheckpointTensors
from gcore_b200.ops import _lib, depth, moe
from gcore_b200.ops import latent_attention as la
from gcore_b200.ops import matrix_memory as mm
from gcore_b200.rollout.engine import SamplingParams
from tests import kedesun_util as ku
from tests.oracle import kedesun as oracle

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


# ---------------------------------------------------------------------------------------------------- latent attention
@DTYPES
@pytest.mark.parametrize("H,dim,rot,vdim,rank,bs", [
    (6, 24, 8, 40, 96, 8), (16, 128, 64, 128, 512, 64), (20, 64, 32, 64, 256, 16), (3, 100, 48, 72, 200, 12), (1, 20, 6, 12, 36, 16),
    (2, 136, 16, 48, 64, 16), (2, 40, 96, 40, 80, 16), (1, 8, 2, 8, 600, 12), (17, 16, 4, 136, 128, 128)])
def test_latent_attention_alone(H, dim, rot, vdim, rank, bs, dtype):
    """Random latents, and per request queries that single out one key: the first, the oldest of a page, the one in front of
    the portion, the newest.  Sizes of every prompt and decode kernel, and of the general one."""
    torch.manual_seed(1)
    dt = DT[dtype]
    segs = [(0, 150), (333, 70), (63, 2), (127, 65), (5, 2), (500, 1), (0, 1), (64, 1), (255, 1)]
    total = [f + l for f, l in segs]
    rows = ku.make_rows(segs, bs, sum((t + bs - 1) // bs for t in total) + 5, 16)
    sp = ku.latent(H, dim, rot, vdim, rank, 0.35 * (dim + rot) ** -0.5, None, base=300.0)
    spec = from_hf_config(ku.conf([sp], 8, 8)).layer_plan.layers[0].mixer
    m, eps = sp["mixer"], 1e-4
    mix = LatentAttentionMixer(spec, 8, eps, dt, "cuda")
    ly = mix.layout
    uk = (torch.randn(H, dim, rank) * rank ** -0.5).to(dt)
    uv = (torch.randn(H, vdim, rank) * rank ** -0.5).to(dt)
    gain = torch.rand(rank) + 0.5
    W = {"q": torch.zeros(H * (dim + rot), 8), "dkv": torch.zeros(rank + rot, 8), "dkv.norm": gain, "g": torch.zeros(H, 8),
         "uk": uk.reshape(-1, rank), "uv": uv.reshape(-1, rank), "o": torch.zeros(8, H * vdim)}
    mix.load(CheckpointTensors(W), "", torch.zeros(mix.columns, 8, device="cuda", dtype=dt),
             torch.zeros(8, mix.out_columns, device="cuda", dtype=dt))
    cache = torch.full((int(rows.tables.max()) + 6, bs, 1, ly.row), 3.0, dtype=dt, device="cuda")
    flat = cache.view(-1, ly.row)
    lead = 16                                           # the mixer's columns need not start the row
    proj = torch.zeros(sum(l for _, l in segs), lead + mix.columns, dtype=dt, device="cuda")
    view, at, keep = proj[:, lead:], 0, []
    for s, (f, l) in enumerate(segs):
        n = f + l
        down, gate = torch.randn(n, rank + rot).to(dt), torch.randn(l, H).to(dt)
        lat = (oracle.rms(down[:, :rank].double(), eps) * gain).to(dt).double()
        kr = oracle.rotate(down[:, rank:].double(), m["rot"], range(n)).to(dt).double()
        k, v = torch.einsum("hdc,nc->nhd", uk.double(), lat), torch.einsum("hvc,nc->nhv", uv.double(), lat)
        q = torch.randn(l, H, dim + rot).to(dt)
        targets = [0, max(0, n - 1 - (n - 1) % bs), max(0, f - 1), n - 1, max(0, (n - 1) // bs * bs - 1)]
        for h in range(H):                              # the last row points at one key in its unrotated part
            j = targets[h % 5]
            q[-1, h, :dim] = (k[j, h] * 60 / k[j, h].pow(2).sum().sqrt()).to(dt)
        p = torch.arange(f)
        old = torch.zeros(f, ly.row, dtype=dt)
        old[:, :rank], old[:, ly.row_rank:ly.row_rank + rot] = lat[:f].to(dt), kr[:f].to(dt)
        where = lambda p, tab=rows.tables[s].cpu(): (tab[p // bs].long() * bs + p % bs).cuda()
        flat[where(p)] = old.cuda()
        qv = view[at:at + l, ly.q:ly.q + H * (ly.dim + ly.row_rot)].view(l, H, -1)
        qv[..., :dim], qv[..., ly.dim:ly.dim + rot] = q[..., :dim].cuda(), q[..., dim:].cuda()
        view[at:at + l, ly.down:ly.down + rank] = down[f:, :rank].cuda()
        view[at:at + l, ly.down + ly.row_rank:ly.down + ly.row_rank + rot] = down[f:, rank:].cuda()
        view[at:at + l, ly.gate:ly.gate + H] = gate.cuda()
        qr = oracle.rotate(q[..., dim:].double(), m["rot"], range(f, n))
        keep.append((at, f, l, lat, kr, k, v, q.double(), qr, gate.double(), where))
        at += l
    out = torch.full((at, mix.out_columns + 8), 7.0, dtype=dt, device="cuda")
    la.latent_attention(view, ly, mix.gain, mix.turns, mix.up_kv, rows, cache, out[:, :mix.out_columns])
    assert (out[:, mix.out_columns:] == 7).all()
    got = out[:, :mix.out_columns].view(at, H, ly.vdim).double().cpu()
    assert not got[..., vdim:].any()
    for at, f, l, lat, kr, k, v, q, qr, gate, where in keep:
        for r in sorted({0, 1, l // 2, l - 2, l - 1} & set(range(l))):
            i = f + r
            s = (torch.einsum("hd,nhd->hn", q[r, :, :dim], k[:i + 1]) + qr[r] @ kr[:i + 1].T) * m["scale"]
            want = torch.einsum("hn,nhv->hv", torch.softmax(s, -1), v[:i + 1]) * torch.sigmoid(gate[r])[:, None]
            err = (got[at + r, :, :vdim] - want).abs().max() / want.abs().max().clamp_min(0.5)
            assert err < (5e-5 if dtype == "float32" else 3e-2), (f, l, r, float(err))
        p = torch.arange(f, f + l)                      # the new rows went to their slots, zero where padded
        stored = flat[where(p)].double().cpu()
        tol = 1e-5 if dtype == "float32" else 2e-2
        assert (stored[:, :rank] - lat[f:]).abs().max() < tol and not stored[:, rank:ly.row_rank].any()
        assert (stored[:, ly.row_rank:ly.row_rank + rot] - kr[f:]).abs().max() < 2 * tol
        assert not stored[:, ly.row_rank + rot:].any()


def test_latent_decode_splits_agree():
    """A long context cut into many splits = the same in one."""
    torch.manual_seed(2)
    lib = _lib.kernels()
    spec = from_hf_config(ku.conf([ku.latent(16, 64, 32, 64, 512, 0.05, None)], 8, 8)).layer_plan.layers[0].mixer
    mix = LatentAttentionMixer(spec, 8, 1e-5, torch.bfloat16, "cuda")
    ly = mix.layout
    mix.up_kv.normal_(0, ly.row_rank ** -0.5)
    mix.gain.fill_(1.0)
    rows = ku.make_rows([(5000, 1), (130, 1)], 64, 90, 2)
    cache = torch.randn(91, 64, 1, ly.row, device="cuda").bfloat16()
    proj = torch.randn(2, mix.columns, device="cuda").bfloat16()
    outs = []
    for target in (0, 1):
        lib.gk_mla_set_target_ctas(target)
        out = torch.empty(2, mix.out_columns, dtype=torch.bfloat16, device="cuda")
        la.latent_attention(proj.clone(), ly, mix.gain, mix.turns, mix.up_kv, rows, cache.clone(), out)
        outs.append(out.float())
    lib.gk_mla_set_target_ctas(0)
    assert (outs[0] - outs[1]).abs().max() < 1e-2 and outs[0].abs().max() > 1e-2


def test_rotation_is_exact_far_out():
    """Positions up to a million, against float64."""
    sp = ku.latent(1, 8, 16, 8, 32, 0.2, None, base=3000.0, factor=4.0, original=50000)
    mix = LatentAttentionMixer(from_hf_config(ku.conf([sp], 8, 8)).layer_plan.layers[0].mixer, 8, 1e-5, torch.float32, "cuda")
    ly, at = mix.layout, [0, 1, 77, 4095, 65537, 262143, 1000003]
    rows = ku.make_rows([(0, 1)] * len(at), 16, 8, 8)
    rows.pos.copy_(torch.tensor(at))
    proj = torch.randn(len(at), mix.columns, device="cuda")
    kr = proj[:, ly.down + ly.row_rank:][:, :16].double().cpu()
    cache = torch.zeros(9, 16, ly.row, device="cuda")
    la._prep(proj, ly, mix.gain, mix.turns, rows, cache, None)
    got = cache.view(-1, ly.row)[rows.slots.long()][:, ly.row_rank:ly.row_rank + 16].double().cpu()
    assert (got - oracle.rotate(kr, sp["mixer"]["rot"], at)).abs().max() < 3e-6


def test_inactive_rows_leave_the_cache_alone():
    spec = from_hf_config(ku.conf([ku.latent(2, 16, 8, 16, 32, 0.2, None)], 8, 8)).layer_plan.layers[0].mixer
    for dt in DT.values():
        mix = LatentAttentionMixer(spec, 8, 1e-5, dt, "cuda")
        rows = ku.make_rows([(9, 1), (20, 1)], 16, 8, 2)
        rows.slots[0], rows.ctx[0] = -1, 0
        cache = torch.zeros(9, 16, 1, mix.layout.row, dtype=dt, device="cuda")
        out = torch.ones(2, mix.out_columns, dtype=dt, device="cuda")
        mix.gain.fill_(1.0)
        la.latent_attention(torch.ones(2, mix.columns, dtype=dt, device="cuda"), mix.layout, mix.gain, mix.turns, mix.up_kv, rows,
                            cache, out)
        assert not out[0].any() and (cache.view(-1, mix.layout.row).abs().sum(-1) > 0).sum() == 1


# ---------------------------------------------------------------------------------------------------- retention
@pytest.mark.parametrize("finish", [0, 1 << 30])     # single tokens: output kernel behind the scan / finished in one launch
@DTYPES
@pytest.mark.parametrize("heads,dim,vdim,true", [(3, 16, 16, 11), (2, 64, 128, 128), (2, 128, 80, 75), (1, 256, 64, 64),
                                                 (2, 144, 208, 208), (1, 320, 32, 32), (1, 32, 528, 520), (4, 48, 64, 50)])
def test_retention_alone(heads, dim, vdim, true, dtype, finish, monkeypatch):
    """Portions and single tokens with decays from nearly nothing to one, carried state and fresh slots."""
    torch.manual_seed(3)
    dt, eps = DT[dtype], 1e-5
    segs = [(0, 300), (70, 130), (0, 2), (40, 7), (128, 128), (3, 129), (0, 1), (9, 1), (200, 1)]
    rows = ku.make_rows(segs, 16, 240, 12)
    ofs = [0, heads * dim, 2 * heads * dim, 2 * heads * dim + heads * vdim]
    decay = [[0.97], [0.6, 1.0], [0.004, 0.9, 0.9995], [0.0, 0.5, 0.999, 1.0]][heads - 1]
    state = mm.MemoryState.allocate(12, heads, dim, vdim, "cuda", gated=False)
    state.S.fill_(99.0)                                  # what earlier requests left
    proj, wants, states = [], [], []
    for s, (f, l) in enumerate(segs):
        pr = torch.randn(l, ofs[3] + heads * vdim).to(dt)
        pr[:, ofs[2]:].view(l, 2 * heads, vdim)[..., true:] = 0
        S = torch.randn(heads, dim, vdim) if f else torch.zeros(heads, dim, vdim)
        S[..., true:] = 0
        if f:
            state.S[int(rows.states[s])] = S.cuda()
        S = S.double() * dim ** -0.5                     # the kernel keeps the keys' factor out of the state
        part = lambda a, n: pr[:, a:a + heads * n].view(l, heads, n).double()
        wants.append(oracle.retention_core(part(ofs[0], dim), part(ofs[1], dim), part(ofs[2], vdim), decay, S))
        states.append(S * dim ** 0.5)
        proj.append(pr)
    monkeypatch.setattr(mm, "FINISH_CTAS", finish)
    raw, output = [], mm._output
    monkeypatch.setattr(mm, "_output", lambda o, *a: raw.append(o.clone()) or output(o, *a))
    y = torch.full((sum(l for _, l in segs), heads * vdim + 16), 5.0, dtype=dt, device="cuda")
    mm.retention(torch.cat(proj).cuda(), *ofs, torch.tensor(decay, device="cuda"), dim ** -0.5, heads, dim, vdim, true, rows,
                 state, eps, y[:, :heads * vdim])
    assert (y[:, heads * vdim:] == 5).all()
    o, at = torch.cat(raw).double().cpu(), 0
    # bf16 inputs are exact in both: what is left is the two-term operands
    tol = 1e-4 if dtype == "float32" else 2e-3
    for s, (f, l) in enumerate(segs):
        if at < o.shape[0]:
            d = (o[at:at + l] - wants[s]).abs().amax(-1) / wants[s].abs().amax()
            assert d.max() < tol, (s, float(d.max()), int(d.amax(-1).argmax()))
        got = state.S[int(rows.states[s])].cpu()
        assert (got - states[s]).abs().max() < tol * states[s].abs().max().clamp_min(1e-2), s
        at += l
    z = torch.cat(proj)[:, ofs[3]:].double()
    o = torch.cat(wants)
    want = (o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / true + eps)).reshape(at, -1) * oracle.silu(z)
    err = (y[:, :heads * vdim].double().cpu() - want).abs()
    assert err.max() < (5e-3 if dtype == "float32" else 0.15) and err.mean() < (1e-5 if dtype == "float32" else 4e-3)


# ---------------------------------------------------------------------------------------------------- feed-forward
@DTYPES
@pytest.mark.parametrize("F,rows", [(8, 1), (52, 7), (384, 130), (1000, 33)])
def test_activations_alone(F, rows, dtype):
    torch.manual_seed(4)
    dt = DT[dtype]
    src, up = (torch.randn(rows, 2 * F + 40) * 3).to(dt).cuda(), F + 24
    dst = torch.full((rows, F + 16), 9.0, dtype=dt, device="cuda")
    logit = torch.randn(rows, 5, device="cuda")
    s = src.double().cpu()
    for kind, want in ((moe.SILU_GATE, oracle.silu(s[:, :F]) * s[:, up:up + F]), (moe.RELU2, torch.relu(s[:, up:up + F]) ** 2)):
        for gated in (False, True):
            moe.activate(kind, src, F, up, dst[:, 8:8 + F], logit[:, 2] if gated else None)
            w = want * torch.sigmoid(logit[:, 2:3].double().cpu()) if gated else want
            assert ((dst[:, 8:8 + F].double().cpu() - w).abs() / w.abs().clamp_min(1)).max() < (1e-5 if dtype == "float32" else 6e-3)
            assert (dst[:, :8] == 9).all() and (dst[:, 8 + F:] == 9).all()
    before = dst.clone()                                 # only the rows in use
    moe.activate(moe.RELU2, src, F, up, dst[:, 8:8 + F], n_rows=torch.tensor([rows // 2], dtype=torch.int32, device="cuda"))
    assert torch.equal(dst[rows // 2:], before[rows // 2:])


@pytest.mark.parametrize("E,K", [(1, 1), (5, 2), (12, 3), (32, 16), (33, 4), (100, 6), (200, 1), (256, 8), (511, 5), (512, 8)])
def test_choice_of_experts_alone(E, K):
    torch.manual_seed(5)
    T = 77
    logits = torch.randn(T, E + 3, device="cuda") * 2
    corr = torch.randn(E, device="cuda") * 0.05
    counts = torch.zeros(E, dtype=torch.int32, device="cuda")
    idx, w, place = moe.choose(logits, E, K, corr, counts)
    want_n = torch.zeros(E, dtype=torch.int64)
    for t in range(T):
        ref = dict(oracle.choose_experts(logits[t, :E].double().cpu(), corr.double().cpu(), K))
        got = dict(zip(idx[t].tolist(), w[t].tolist()))
        assert set(got) == set(ref), t
        assert all(abs(got[e] - ref[e]) < 1e-5 for e in ref)
        for e in ref:
            want_n[e] += 1
    assert torch.equal(counts.cpu().long(), want_n)
    rows, dest, off = moe.expert_rows(torch.randn(T, 16, device="cuda"), counts, idx, place)
    n = torch.cat([torch.zeros(1, dtype=torch.int64), ((want_n + 127) // 128 * 128).cumsum(0)])
    assert torch.equal(off.cpu().long(), n) and int(n[-1]) <= rows.shape[0] and dest.unique().numel() == T * K


@DTYPES
@pytest.mark.parametrize("T,E,K,width", [(1, 1, 1, 8), (8, 12, 2, 200), (128, 33, 5, 1000), (3, 512, 8, 4096), (40, 64, 4, 11264),
                                         (129, 9, 2, 64)])
def test_routing_from_the_tokens(T, E, K, width, dtype):
    """One launch for few tokens, product and choice for many: the same logits and choice."""
    torch.manual_seed(8)
    h, router = torch.randn(T, width).to(DT[dtype]), (torch.randn(E + 1, width) * width ** -0.5 * 2).to(DT[dtype])
    corr, counts = torch.randn(E) * 0.01, torch.zeros(E, dtype=torch.int32, device="cuda")
    logits, (idx, w, place) = moe.route_tokens(h.cuda(), router.cuda(), E, K, corr.cuda(), counts)
    want = h.double() @ router.double().T
    assert (logits.double().cpu() - want).abs().max() < 2e-5 and int(counts.sum()) == T * K
    got = logits.double().cpu()
    for t in range(T):
        ref = dict(oracle.choose_experts(got[t, :E], corr.double(), K))
        assert set(idx[t].tolist()) == set(ref)
        assert all(abs(x - ref[e]) < 1e-5 for e, x in zip(idx[t].tolist(), w[t].tolist()))
    flat = idx * 1000 + place
    assert flat.unique().numel() == T * K and (place < counts[idx]).all()


@DTYPES
@pytest.mark.parametrize("T,E,K,F,width", [(1, 5, 2, 24, 48), (8, 64, 4, 128, 256), (300, 12, 3, 72, 200), (130, 7, 1, 136, 64),
                                           (40, 200, 6, 16, 32)])
def test_routed_experts_alone(T, E, K, F, width, dtype):
    """Uneven loads, one expert that takes every token, one that takes none."""
    torch.manual_seed(6)
    dt = DT[dtype]
    h = torch.randn(T, width).to(dt)
    logits, corr = torch.randn(T, E) * 2, torch.randn(E) * 0.05
    corr[0], corr[-1] = 9.0, -9.0
    up, down = (torch.randn(E, F, width) * width ** -0.5).to(dt), (torch.randn(E, width, F) * F ** -0.5).to(dt)
    counts = torch.zeros(E, dtype=torch.int32, device="cuda")
    choice = moe.choose(logits.cuda(), E, K, corr.cuda(), counts)
    rows, dest, w = moe.routed_experts(h.cuda(), choice, up.cuda(), down.cuda(), counts)
    got = (rows[dest.long()].double() * w[:, :, None].double()).sum(1).cpu()
    assert int(counts[0]) == T and int(counts[-1]) == 0
    for t in range(T):
        want = sum(x * (down[e].double() @ torch.relu(up[e].double() @ h[t].double()) ** 2)
                   for e, x in oracle.choose_experts(logits[t].double(), corr.double(), K))
        assert (got[t] - want).abs().max() < (1e-5 if dtype == "float32" else 2e-2) * want.abs().max().clamp_min(1), t


# ---------------------------------------------------------------------------------------------------- residual step
@DTYPES
@pytest.mark.parametrize("width,pad", [(44, 48), (192, 192), (1000, 1000), (2048, 2048), (5000, 5000), (9000, 9000)])
def test_depth_average_alone(width, pad, dtype):
    torch.manual_seed(7)
    dt, T, eps, n = DT[dtype], 5, 1e-3, 6
    c = lambda t: torch.nn.functional.pad(t, (0, pad - width)).contiguous().cuda()
    hist = torch.zeros(n + 2, T, pad, device="cuda")
    past = [torch.randn(T, width) for _ in range(n)]
    for j, p in enumerate(past):
        hist[j] = c(p)
    x, y, avg, gain = torch.randn(T, width), torch.randn(T, width).to(dt), torch.randn(n + 1), torch.rand(width) + 0.5
    er, dest = torch.randn(40, width).to(dt), torch.randperm(40)[:T * 3].view(T, 3).int()
    w = torch.rand(T, 3)
    for routed in (None, (c(er), dest.cuda(), w.cuda())):
        for keep in (True, False):
            hist[n], xg = 7.0, c(x)
            h = depth.add_layer(hist, n, xg, c(y), avg.cuda(), width, eps, xg, c(gain), routed, keep=keep)
            new = x.double() + y.double()
            if routed:
                new = new + (er.double()[dest.long()] * w[:, :, None]).sum(1)
            want = oracle.depth_average(avg.double(), [p.double() for p in past] + [new])
            assert (xg[:, :width].cpu() - want).abs().max() < 2e-5 and not xg[:, width:].any()
            assert (hist[n, :, :width].cpu() - new).abs().max() < 1e-5 if keep else (hist[n] == 7).all()
            ref = oracle.rms(want, eps) * gain
            assert (h[:, :width].cpu().double() - ref).abs().max() < (2e-5 if dtype == "float32" else 3e-2)
    assert depth.add_layer(hist, 1, hist[0], c(y), avg.cuda(), width, eps, xg) is None
    assert (xg[:, :width].cpu() - (avg[0] * past[0] + avg[1] * (past[0] + y.float()))).abs().max() < 1e-5


# ---------------------------------------------------------------------------------------------------- engine
@DTYPES
@pytest.mark.parametrize("which", ["uneven", "round"])
def test_portions_and_decoding_match_whole_sequences(which, dtype):
    c = ku.uneven_conf() if which == "uneven" else ku.round_conf()
    W = oracle.random_weights(c, seed=5)
    eng = ku.make_engine(c, W, dtype, "cuda")
    for n, seed in ((1, 1), (2, 2), (150, 3), (333, 4)):
        seq = ku.tokens(n, c["vocab"], seed)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [64, 1], [15, 17, 1, 1, 100, 2]):
            if cuts == [1] and n > 200 or cuts == [2] and n < 200:
                continue
            ku.assert_close(ku.run_alone(eng, seq, cuts), want, dtype, (n, cuts))
    assert eng.get_load()["free_blocks"] == eng.num_blocks


@DTYPES
@pytest.mark.parametrize("block", [8, 64])
def test_mixed_batches_on_reused_pages_and_slots(dtype, block):
    c = ku.round_conf()
    W = oracle.random_weights(c, seed=6)
    eng = ku.make_engine(c, W, dtype, "cuda", kv_block_size=block, num_kv_blocks=4 * 256 // block, max_model_len=256)
    seqs = [ku.tokens(n, c["vocab"], 20 + n) for n in (200, 31, 64, 1, 129, 65, 90, 17, 240)]
    for s, got in zip(seqs, ku.run_mixed(eng, seqs, [1, 1, 2, 3, 16, 63, 64, 65, 100], seed=7)):
        ku.assert_close(got, oracle.forward(W, c, s), dtype)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_the_batch_does_not_matter():
    """bf16 logits of one request alone and in a batch of others differ by rounding only."""
    c = ku.round_conf()
    W = oracle.random_weights(c, seed=12)
    eng = ku.make_engine(c, W, "bfloat16", "cuda", max_model_len=256)
    seqs = [ku.tokens(n, c["vocab"], 70 + n) for n in (120, 77, 33, 5)]
    for s, got in zip(seqs, ku.run_mixed(eng, seqs, [1, 2, 30, 64], seed=8)):
        ku.assert_close(got, ku.run_alone(eng, s, [len(s)]).double(), "bfloat16")


def test_true_32_bit_whatever_the_matrix_mode():
    """The 32-bit engine stays exact when the process allows TF32."""
    c = ku.round_conf()
    W = oracle.random_weights(c, seed=8)
    eng = ku.make_engine(c, W, "float32", "cuda")
    seq = ku.tokens(70, c["vocab"], 9)
    torch.backends.cuda.matmul.allow_tf32 = True
    try:
        got = ku.run_alone(eng, seq, [40, 1])
    finally:
        torch.backends.cuda.matmul.allow_tf32 = False
    ku.assert_close(got, oracle.forward(W, c, seq))


@DTYPES
def test_greedy_generation_through_the_scheduler(dtype):
    """generate(): captured decode graphs, more requests than slots, prompts longer than a prefill step, samples that
    share a prompt - every token is the plain implementation's choice (or ties with it within rounding)."""
    c = ku.uneven_conf() if dtype == "float32" else ku.round_conf()
    W = oracle.random_weights(c, seed=10)
    eng = ku.make_engine(c, W, dtype, "cuda", max_prefill_tokens=50, sync_interval=3, max_model_len=256)
    prompts = [ku.tokens(n, c["vocab"], 40 + n) for n in (1, 5, 33, 120, 64)]
    reqs = eng.generate(prompts, SamplingParams(max_new_tokens=40, greedy=True), n=2)
    assert eng.stats["graph_replays"] > 0
    for k, r in enumerate(reqs):
        assert len(r.out_tokens) == 40
        if dtype == "float32":
            assert r.out_tokens == reqs[k // 2 * 2].out_tokens
        if k % 2 == 0:
            lg = oracle.forward(W, c, r.prompt + r.out_tokens)[len(r.prompt) - 1:-1]
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert gap.max() < (1e-4 if dtype == "float32" else 0.25) * lg.std(), float(gap.max())
            lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert (lp - torch.tensor(r.out_logprobs)).abs().max() < (1e-3 if dtype == "float32" else 0.5) * lg.std().clamp_min(1)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_long_decoding_keeps_the_state():
    c = ku.conf([ku.retention(2, 32, 64, ku.dense(64), decay=[0.9, 0.998]), ku.latent(4, 32, 8, 32, 64, 0.15, ku.dense(64))],
                64, 128)
    W = oracle.random_weights(c, seed=11)
    eng = ku.make_engine(c, W, "bfloat16", "cuda", max_model_len=1024)
    seq = ku.tokens(600, c["vocab"], 12)
    ku.assert_close(ku.run_alone(eng, seq, [20] + [1] * 580), oracle.forward(W, c, seq), "bfloat16")


def _checkpoint(path, c, seed):
    from safetensors.torch import save_file
    W = oracle.random_weights(c, seed=seed)
    save_file({k: v.contiguous() for k, v in W.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(c))
    return W


def test_command_line_generates_from_a_checkpoint_folder(tmp_path):
    from gcore_b200.entry import lm_infer
    c = ku.round_conf()
    W = _checkpoint(tmp_path, c, 13)
    prompts = [ku.tokens(n, c["vocab"], n) for n in (7, 20)]
    (tmp_path / "p.jsonl").write_text("".join(json.dumps({"prompt_token_ids": p}) + "\n" for p in prompts))
    out = tmp_path / "o.jsonl"
    lm_infer.main([f"checkpoint.load_ckpt_path={tmp_path}", f"+task.infer.prompts={tmp_path}/p.jsonl",
                   f"+task.infer.out={out}", "+task.infer.greedy=true"])
    got = [json.loads(l) for l in out.read_text().splitlines()]
    assert [g["prompt_length"] for g in got] == [7, 20]
    for g, p in zip(got, prompts):
        assert len(g["tokens"]) == len(p) + 128 and g["tokens"][:len(p)] == p
        lg = oracle.forward(W, c, g["tokens"][:len(p) + 20])[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(g["tokens"][len(p):len(p) + 20])[:, None])[:, 0]
        assert gap.max() < 0.25 * lg.std()


def test_trace_replay_through_the_executable_entry(tmp_path):
    import numpy as np

    from gcore_b200.entry import trace_run
    c = ku.uneven_conf()
    W = _checkpoint(tmp_path, c, 14)
    eng = trace_run.build_engine(str(tmp_path), "float32", 128, torch.device("cuda", 0))
    a, b = ku.tokens(40, c["vocab"], 1), ku.tokens(9, c["vocab"], 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[1:], want=[])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=b, want=[8]), dict(id="a", tokens=a[30:], want=[9])], end=["a", "c"])]
    said = []
    trace_run.replay(eng, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    la_, lb = oracle.forward(W, c, a), oracle.forward(W, c, b)
    for n, want in ((0, torch.stack([la_[0], la_[29], lb[0]])), (2, torch.stack([lb[8], la_[39]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"]).copy())
        ku.assert_close(got, want)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_serving_benchmark_runs_on_a_small_size():
    from gcore_b200.tools import serve_bench as sb
    from gcore_b200.tools import serve_bench_kedesun as sk
    s = dict(width=256, heads=4, dim=128, rot=64, vdim=128, rank=256, rh=2, rk=64, rv=128, ff=512, experts=8, top=2, eff=192,
             layers=4)
    for kind in ("kedesun", "latent"):
        eng = sb.build(kind, s, 512, 4)
        assert sb.prefill_step(eng, 2, 130, 2) > 0 and sb.decode_step(eng, 4, 200, 2) > 0
        assert sk.decode_bytes(kind, s, eng, 4, 200) > 0
    table = sk.kernel_table(s, 2, 130, 4, 200)
    assert {r[0] for r in table} == {"prefill", "decode"} and all(r[2] > 0 for r in table)

"""Lobutar on the GPU: every kernel alone against the plain implementation, then the engine - portions, mixed batches, freed
pages and slots, long decoding, generation - against whole sequences of the plain implementation."""
import json

import pytest
import torch

from gcore_b200.models.config import from_hf_config
from gcore_b200.models.plan_decoder import CheckpointTensors
from gcore_b200.models.plan_modules import DifferentialAttentionMixer, LatentAttentionMixer
from gcore_b200.ops import _lib, moe
from gcore_b200.ops import diff_attention as da
from gcore_b200.ops import latent_attention as la
from gcore_b200.ops import streams as hc
from gcore_b200.rollout.engine import SamplingParams
from tests import lobutar_util as lu
from tests.oracle import lobutar as oracle

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def _spec(entry):
    return from_hf_config(lu.conf([entry], 8, 8)).layer_plan.layers[0].mixer


def _pool(rows, bs, row, dt, fill):
    """A cache for the rows' pages, filled with what earlier requests left, and where a request's positions lie in it."""
    cache = torch.full((int(rows.tables.max()) + 6, bs, row), fill, dtype=dt, device="cuda")
    tabs = rows.tables.cpu()
    return cache, lambda s, p: (tabs[s][p // bs].long() * bs + p % bs).cuda()


# ---------------------------------------------------------------------------------------------- differential attention
SEGS = [(0, 150), (333, 70), (63, 2), (127, 65), (5, 2), (500, 1), (0, 1), (64, 1), (255, 1), (31, 1)]


@DTYPES
@pytest.mark.parametrize("H,G,dim,vdim,rot,bs", [
    (6, 2, 40, 72, 8, 16), (16, 4, 64, 128, 64, 64), (5, 5, 24, 40, 10, 8), (12, 1, 128, 128, 32, 32), (3, 3, 100, 60, 100, 128),
    (20, 2, 56, 200, 6, 16), (2, 1, 128, 256, 128, 64), (2, 2, 136, 48, 16, 16), (4, 2, 20, 264, 4, 16), (4, 2, 32, 64, 12, 12)])
def test_differential_attention_alone(H, G, dim, vdim, rot, bs, dtype):
    """Random keys, and in the last row of every request queries that single out one key per map - the first, the last of a
    page, the one in front of the portion, the newest - another one in each map.  Sizes of every prompt and decode kernel, and
    of the general one."""
    torch.manual_seed(1)
    dt, eps = DT[dtype], 1e-4
    total = [f + l for f, l in SEGS]
    rows = lu.make_rows(SEGS, bs, sum((t + bs - 1) // bs for t in total) + 5, 16)
    entry = lu.attention(H, G, dim, vdim, rot, 0.4 * dim ** -0.5, 0.35, None, base=300.0)
    m = entry["mixer"]
    mix = DifferentialAttentionMixer(_spec(entry), 8, eps, dt, "cuda")
    ly = mix.layout
    W = {f"{n}": torch.zeros(r, 8) for n, r in (("q", 2 * H * dim), ("k", 2 * G * dim), ("v", G * vdim), ("g", H))}
    W.update({n + ".b": torch.zeros(W[n].shape[0]) for n in "qkv"}, o=torch.zeros(8, H * vdim))
    W.update({n: torch.randn(dim) * 0.5 * dim ** -0.5 for n in ("lq1", "lk1", "lq2", "lk2")})
    mix.load(CheckpointTensors(W), "", torch.zeros(mix.columns, 8, device="cuda", dtype=dt),
             torch.zeros(8, mix.out_columns, device="cuda", dtype=dt), torch.zeros(mix.columns, device="cuda"))
    lam = oracle.difference_weight(*(W[n].double() for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    assert float(mix.lam) == pytest.approx(lam, rel=1e-6)
    cache, where = _pool(rows, bs, ly.row, dt, 3.0)
    flat = cache.view(-1, ly.row)
    lead = 16                                           # the mixer's columns need not start the row
    proj = torch.zeros(sum(l for _, l in SEGS), lead + mix.columns, dtype=dt, device="cuda")
    view, at, keep = proj[:, lead:], 0, []
    for s, (f, l) in enumerate(SEGS):
        n = f + l
        k0, v, gate = torch.randn(n, G, 2, dim).to(dt), torch.randn(n, G, vdim).to(dt), torch.randn(l, H).to(dt)
        q = torch.randn(l, H, 2, dim).to(dt)
        k = oracle.rotate(k0.double(), m["rot"], range(n)).to(dt).double()
        targets = [0, max(0, n - 1 - (n - 1) % bs), max(0, f - 1), n - 1, max(0, (n - 1) // bs * bs - 1)]
        back = oracle.rotate                            # rotating the query back makes it point at the rotated key
        for h in range(H):
            for i in range(2):
                key = k[targets[(h + 2 * i) % 5], h // (H // G), i]
                want = (key * 60 / key.pow(2).sum().sqrt())[None]
                q[-1, h, i] = (2 * torch.cat([want[:, :rot] * 0, want[:, rot:]], -1) if rot < dim else
                               _unrotate(want, m["rot"], n - 1))[0].to(dt)
        old = torch.cat([_pad(k[:f].to(dt), ly.dim).flatten(1), _pad(v[:f], ly.vdim).flatten(1)], 1)
        flat[where(s, torch.arange(f))] = old.cuda()
        sl = view[at:at + l]
        sl[:, ly.q:ly.q + 2 * H * ly.dim] = _pad(q, ly.dim).flatten(1).cuda()
        sl[:, ly.k:ly.k + 2 * G * ly.dim] = _pad(k0[f:], ly.dim).flatten(1).cuda()
        sl[:, ly.v:ly.v + G * ly.vdim] = _pad(v[f:], ly.vdim).flatten(1).cuda()
        sl[:, ly.gate:ly.gate + H] = gate.cuda()
        keep.append((s, at, f, l, back(q.double(), m["rot"], range(f, n)), k, v.double(), gate.double()))
        at += l
    out = torch.full((at, mix.out_columns + 8), 7.0, dtype=dt, device="cuda")
    da.differential_attention(view, ly, mix.turns, mix.lam, rows, cache, out[:, :mix.out_columns])
    _lib.check_device_errors()
    assert (out[:, mix.out_columns:] == 7).all()
    got = out[:, :mix.out_columns].view(at, H, ly.vdim).double().cpu()
    assert not got[..., vdim:].any()
    for s, at, f, l, qr, k, v, gate in keep:
        for r in sorted({0, 1, l // 2, l - 2, l - 1} & set(range(l))):
            n, g = f + r + 1, torch.arange(H) // (H // G)
            sc = torch.einsum("hmd,nhmd->hmn", qr[r], k[:n, g]) * m["scale"]
            a = torch.einsum("hmn,nhv->hmv", torch.softmax(sc, -1), v[:n, g])
            want = oracle.combine_maps(a[:, 0], a[:, 1], lam, m["diff"], eps) * torch.sigmoid(gate[r])[:, None]
            err = (got[at + r, :, :vdim] - want).abs().max() / want.abs().max().clamp_min(0.5)
            assert err < (2e-4 if dtype == "float32" else 6e-2), (f, l, r, float(err))
        stored = flat[where(s, torch.arange(f, f + l))].double().cpu()     # the new rows went to their slots, zero where padded
        ks, vs = stored[:, :ly.value_offset].view(l, G, 2, ly.dim), stored[:, ly.value_offset:].view(l, G, ly.vdim)
        assert (ks[..., :dim] - k[f:]).abs().max() < (1e-5 if dtype == "float32" else 4e-2)
        assert torch.equal(vs[..., :vdim], v[f:]) and not ks[..., dim:].any() and not vs[..., vdim:].any()


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1]))


def _unrotate(x, rot, position):
    return oracle.rotate(x, dict(rot, base=rot["base"]), [-position])


def _diff_mixer(entry, dt=torch.bfloat16):
    mix = DifferentialAttentionMixer(_spec(entry), 8, 1e-5, dt, "cuda")
    mix.lam.fill_(0.6)
    return mix


@pytest.mark.parametrize("vdim", [64, 128, 232])
def test_differential_decode_splits_agree(vdim):
    """A long context cut into many splits = the same in one."""
    torch.manual_seed(2)
    lib = _lib.kernels()
    mix = _diff_mixer(lu.attention(12, 4, 64, vdim, 32, 0.1, 0.3, None))
    ly = mix.layout
    rows = lu.make_rows([(5000, 1), (130, 1), (127, 1)], 64, 90, 3)
    cache = torch.randn(91, 64, ly.row, device="cuda").bfloat16()
    proj = torch.randn(3, mix.columns, device="cuda").bfloat16()
    outs = []
    for target in (0, 1, 60):
        lib.gk_diff_set_target_ctas(target)
        out = torch.empty(3, mix.out_columns, dtype=torch.bfloat16, device="cuda")
        da.differential_attention(proj.clone(), ly, mix.turns, mix.lam, rows, cache.clone(), out)
        outs.append(out.float())
    lib.gk_diff_set_target_ctas(0)
    assert all((o - outs[0]).abs().max() < 2e-2 * outs[0].abs().max() for o in outs[1:])


def test_rotation_is_exact_far_out():
    """Positions up to a million, against float64."""
    entry = lu.attention(1, 1, 20, 8, 16, 0.2, 0.1, None, base=3000.0)
    mix = _diff_mixer(entry, torch.float32)
    ly, at = mix.layout, [0, 1, 77, 4095, 65537, 262143, 1000003]
    rows = lu.make_rows([(0, 1)] * len(at), 16, 8, 8)
    rows.pos.copy_(torch.tensor(at))
    proj = torch.randn(len(at), mix.columns, device="cuda")
    k = proj[:, ly.k:ly.k + 2 * ly.dim].view(-1, 2, ly.dim).double().cpu()
    q = proj[:, ly.q:ly.q + 2 * ly.dim].view(-1, 2, ly.dim).double().cpu()
    cache = torch.zeros(9, 16, ly.row, device="cuda")
    da._append(proj, ly, mix.turns, rows, 0, len(at), cache)
    got = cache.view(-1, ly.row)[rows.slots.long()][:, :2 * ly.dim].view(-1, 2, ly.dim).double().cpu()
    assert (got - oracle.rotate(k, entry["mixer"]["rot"], at)).abs().max() < 3e-6
    q2 = proj[:, ly.q:ly.q + 2 * ly.dim].view(-1, 2, ly.dim).double().cpu()
    assert (q2 - oracle.rotate(q, entry["mixer"]["rot"], at)).abs().max() < 3e-6


def test_inactive_rows_leave_the_cache_alone():
    for dt in DT.values():
        for entry, cls in ((lu.attention(2, 1, 16, 24, 8, 0.2, 0.3, None), DifferentialAttentionMixer),
                           (lu.latent(2, 16, 8, 16, 32, 7, 0.2, None), LatentAttentionMixer)):
            mix = cls(_spec(entry), 8, 1e-5, dt, "cuda")
            for p in (getattr(mix, "gain", None), getattr(mix, "lam", None)):
                if p is not None:
                    p.fill_(0.5)
            rows = lu.make_rows([(9, 1), (20, 1)], 16, 8, 2)
            rows.slots[0], rows.ctx[0] = -1, 0
            cache = torch.zeros(9, 16, *mix.cache_shape(), dtype=dt, device="cuda")
            out = torch.ones(2, mix.out_columns, dtype=dt, device="cuda")
            mix(torch.ones(2, mix.columns, dtype=dt, device="cuda"), rows, cache, None, out)
            assert not out[0].any() and (cache.view(-1, mix.layout.row).abs().sum(-1) > 0).sum() == 1


# ------------------------------------------------------------------------------- latent attention: window, sink, gate
@DTYPES
@pytest.mark.parametrize("H,dim,rot,vdim,rank,bs,window", [
    (6, 24, 8, 40, 96, 8, 61), (16, 128, 64, 128, 512, 64, 128), (20, 64, 32, 64, 256, 16, 33), (3, 100, 48, 72, 200, 12, 64),
    (1, 20, 6, 12, 36, 16, 1), (2, 136, 16, 48, 64, 16, 65), (2, 40, 96, 40, 80, 16, 2), (1, 8, 2, 8, 600, 12, 300),
    (5, 16, 32, 32, 100, 64, 4000)])
def test_window_sink_and_gate_alone(H, dim, rot, vdim, rank, bs, window, dtype):
    """Queries that single out the key just inside the window, the one just outside it, the newest and the oldest; sinks from
    nothing to everything; a gate per element."""
    torch.manual_seed(3)
    dt, eps = DT[dtype], 1e-4
    total = [f + l for f, l in SEGS]
    rows = lu.make_rows(SEGS, bs, sum((t + bs - 1) // bs for t in total) + 5, 16, windows=(window,))
    entry = lu.latent(H, dim, rot, vdim, rank, window, 0.35 * (dim + rot) ** -0.5, None, base=300.0)
    m = entry["mixer"]
    mix = LatentAttentionMixer(_spec(entry), 8, eps, dt, "cuda")
    ly = mix.layout
    uk, uv = (torch.randn(H, dim, rank) * rank ** -0.5).to(dt), (torch.randn(H, vdim, rank) * rank ** -0.5).to(dt)
    gain, sink = torch.rand(rank) + 0.5, torch.tensor([0.0, 3.0, 12.0, -30.0, 40.0])[torch.arange(H) % 5]
    W = {"q": torch.zeros(H * (dim + rot), 8), "dkv": torch.zeros(rank + rot, 8), "dkv.norm": gain, "sink": sink,
         "g": torch.zeros(H * vdim, 8), "uk": uk.reshape(-1, rank), "uv": uv.reshape(-1, rank), "o": torch.zeros(8, H * vdim)}
    mix.load(CheckpointTensors(W), "", torch.zeros(mix.columns, 8, device="cuda", dtype=dt),
             torch.zeros(8, mix.out_columns, device="cuda", dtype=dt))
    cache, where = _pool(rows, bs, ly.row, dt, 3.0)
    flat = cache.view(-1, ly.row)
    view = torch.zeros(sum(l for _, l in SEGS), mix.columns, dtype=dt, device="cuda")
    at, keep = 0, []
    for s, (f, l) in enumerate(SEGS):
        n = f + l
        down, gate = torch.randn(n, rank + rot).to(dt), torch.randn(l, H, vdim).to(dt)
        lat = (oracle.rms(down[:, :rank].double(), eps) * gain).to(dt).double()
        kr = oracle.rotate(down[:, rank:].double(), m["rot"], range(n)).to(dt).double()
        k, v = torch.einsum("hdc,nc->nhd", uk.double(), lat), torch.einsum("hvc,nc->nhv", uv.double(), lat)
        q = torch.randn(l, H, dim + rot).to(dt)
        for r in {0, l // 2, l - 1}:
            i = f + r
            spots = [max(0, i - window + 1), max(0, i - window), i, 0]
            for h in range(H):                          # points at one key in its unrotated part
                j = spots[(h + r) % 4]
                q[r, h, :dim] = (k[j, h] * 60 / k[j, h].pow(2).sum().sqrt()).to(dt)
        old = torch.zeros(f, ly.row, dtype=dt)
        old[:, :rank], old[:, ly.row_rank:ly.row_rank + rot] = lat[:f].to(dt), kr[:f].to(dt)
        flat[where(s, torch.arange(f))] = old.cuda()
        sl = view[at:at + l]
        sl[:, ly.q:ly.q + H * (ly.dim + ly.row_rot)] = torch.cat(
            [_pad(q[..., :dim], ly.dim), _pad(q[..., dim:], ly.row_rot)], -1).flatten(1).cuda()
        sl[:, ly.down:ly.down + rank] = down[f:, :rank].cuda()
        sl[:, ly.down + ly.row_rank:ly.down + ly.row_rank + rot] = down[f:, rank:].cuda()
        sl[:, ly.gate:ly.gate + H * ly.vdim] = _pad(gate, ly.vdim).flatten(1).cuda()
        qr = oracle.rotate(q[..., dim:].double(), m["rot"], range(f, n))
        keep.append((s, at, f, l, lat, kr, k, v, q.double(), qr, gate.double()))
        at += l
    out = torch.full((at, mix.out_columns + 8), 7.0, dtype=dt, device="cuda")
    la.latent_attention(view, ly, mix.gain, mix.turns, mix.up_kv, rows, cache, out[:, :mix.out_columns], mix.sinks)
    _lib.check_device_errors()
    assert (out[:, mix.out_columns:] == 7).all()
    got = out[:, :mix.out_columns].view(at, H, ly.vdim).double().cpu()
    assert not got[..., vdim:].any()
    for s, at, f, l, lat, kr, k, v, q, qr, gate in keep:
        for r in sorted({0, 1, l // 2, l - 2, l - 1} & set(range(l))):
            j = list(oracle.visible(f + r, window))
            sc = (torch.einsum("hd,nhd->hn", q[r, :, :dim], k[j]) + qr[r] @ kr[j].T) * m["scale"]
            w = torch.stack([oracle.softmax_with_sink(sc[h], sink[h].double()) for h in range(H)])
            want = torch.einsum("hn,nhv->hv", w, v[j]) * torch.sigmoid(gate[r])
            err = (got[at + r, :, :vdim] - want).abs().max() / want.abs().max().clamp_min(0.5)
            assert err < (5e-5 if dtype == "float32" else 5e-2), (f, l, r, float(err))
        stored = flat[where(s, torch.arange(f, f + l))].double().cpu()
        assert (stored[:, :rank] - lat[f:]).abs().max() < (1e-5 if dtype == "float32" else 4e-2)


def test_window_decode_splits_agree():
    """Many splits of a window that starts in the middle of a page = one."""
    torch.manual_seed(4)
    lib = _lib.kernels()
    mix = LatentAttentionMixer(_spec(lu.latent(16, 64, 32, 64, 512, 1500, 0.05, None)), 8, 1e-5, torch.bfloat16, "cuda")
    ly = mix.layout
    mix.up_kv.normal_(0, ly.row_rank ** -0.5)
    mix.gain.fill_(1.0)
    mix.sinks.fill_(2.0)
    rows = lu.make_rows([(3000, 1), (130, 1), (1499, 1), (1500, 1)], 64, 120, 4)
    cache = torch.randn(121, 64, ly.row, device="cuda").bfloat16()
    proj = torch.randn(4, mix.columns, device="cuda").bfloat16()
    outs = []
    for target in (0, 1):
        lib.gk_mla_set_target_ctas(target)
        out = torch.empty(4, mix.out_columns, dtype=torch.bfloat16, device="cuda")
        mix(proj.clone(), rows, cache.clone(), None, out)
        outs.append(out.float())
    lib.gk_mla_set_target_ctas(0)
    assert (outs[0] - outs[1]).abs().max() < 1e-2 and outs[0].abs().max() > 1e-2


# ---------------------------------------------------------------------------------------------------- residual streams
@DTYPES
@pytest.mark.parametrize("S,width,pad", [(1, 44, 48), (2, 200, 200), (3, 1000, 1000), (4, 2048, 2048), (5, 44, 48), (8, 520, 520),
                                         (16, 1500, 1504), (4, 9000, 9000)])
def test_stream_mixing_alone(S, width, pad, dtype):
    torch.manual_seed(5)
    dt, T, eps, V = DT[dtype], 5, 1e-3, 31
    c = lambda t: _pad(t, pad).contiguous().cuda()
    embed, gain, read, write = torch.randn(V, width).to(dt), torch.rand(width) + 0.5, torch.randn(S), torch.randn(S)
    mix, tok = torch.randn(S, S), torch.tensor([0, 30, 7, 7, 12])
    tol = 3e-5 if dtype == "float32" else 3e-2
    x, h = hc.embed_rows(tok.cuda(), c(embed), S, read.cuda(), c(gain), width, eps)
    e = embed[tok].double()
    assert all(torch.equal(x[:, s, :width].cpu().double(), e) for s in range(S))
    ref = oracle.rms(oracle.read_streams(read.double(), [e] * S), eps) * gain
    assert (h[:, :width].double().cpu() - ref).abs().max() < tol
    streams = torch.randn(S, T, width)
    y, er, dest = torch.randn(T, width).to(dt), torch.randn(40, width).to(dt), torch.randperm(40)[:T * 3].view(T, 3).int()
    w = torch.rand(T, 3)
    part = (er.double()[dest.long()] * w[:, :, None]).sum(1)
    for yy, routed in ((y, None), (y, (c(er), dest.cuda(), w.cuda())), (None, (c(er), dest.cuda(), w.cuda()))):
        add = (yy.double() if yy is not None else 0) + (part if routed else 0)
        new = oracle.write_streams(mix.double(), write.double(), streams.double(), add)
        for rd in (read, None):
            for keep in (True, False):
                xg = c(streams.transpose(0, 1))
                total = torch.full((T, pad), 9.0, device="cuda")
                h = hc.connect(xg, None if yy is None else c(yy), mix.cuda(), write.cuda(), width, eps,
                               None if rd is None else rd.cuda(), c(gain), routed, total=total, keep=keep)
                u = oracle.read_streams(rd.double(), new) if rd is not None else new.sum(0)
                want = new if keep else streams.double()
                assert (xg[..., :width].cpu() - want.transpose(0, 1)).abs().max() < 2e-5 and not xg[..., width:].any()
                assert (total[:, :width].cpu() - u).abs().max() < 5e-5
                assert (h[:, :width].double().cpu() - oracle.rms(u, eps) * gain).abs().max() < tol
    assert hc.connect(xg, c(y), mix.cuda(), write.cuda(), width, eps) is None


# ---------------------------------------------------------------------------------------------------- experts
ROUTERS = [(8, 2, 4, 2, 1.5), (6, 2, 6, 3, 1.0), (1, 1, 1, 1, 0.3), (32, 4, 32, 7, 2.0), (33, 5, 3, 1, 1.0), (64, 6, 8, 4, 2.5),
           (200, 8, 10, 3, 1.0), (512, 16, 32, 2, 0.7), (12, 3, 2, 2, 1.1), (100, 7, 1, 1, 1.0)]


@pytest.mark.parametrize("E,K,groups,keep,scale", ROUTERS)
def test_grouped_choice_alone(E, K, groups, keep, scale):
    """Also with choice scores below zero, where a group that is out must not come back as a zero."""
    torch.manual_seed(6)
    T = 77
    router = dict(experts=E, top=K, scale=scale, groups=dict(count=groups, keep=keep))
    for shift in (0.0, -3.0):
        logits = torch.randn(T, E, device="cuda") * 2
        corr = torch.randn(E, device="cuda") * 0.3 + shift
        counts = torch.zeros(E, dtype=torch.int32, device="cuda")
        idx, w, place = moe.choose(logits, E, K, corr, counts, sigmoid=True, norm=False, scale=scale, groups=groups, keep=keep)
        assert int(counts.sum()) == T * K
        for t in range(T):
            ref = dict(oracle.choose_experts(logits[t].double().cpu(), corr.double().cpu(), router))
            got = dict(zip(idx[t].tolist(), w[t].tolist()))
            assert set(got) == set(ref) and all(abs(got[e] - ref[e]) < 1e-5 for e in ref), t


@DTYPES
@pytest.mark.parametrize("T", [1, 40, 129])
def test_gated_experts_from_the_tokens(T, dtype):
    """Router (one launch for few tokens, product and choice for many), gated experts, weights that do not sum to one."""
    torch.manual_seed(7)
    dt, E, K, F, width = DT[dtype], 24, 4, 40, 200
    how = dict(sigmoid=True, norm=False, scale=1.8, groups=6, keep=3)
    h, router = torch.randn(T, width).to(dt), (torch.randn(E, width) * width ** -0.5 * 2).to(dt)
    up, down = (torch.randn(E, 2 * F, width) * width ** -0.5).to(dt), (torch.randn(E, width, F) * F ** -0.5).to(dt)
    corr, counts = torch.randn(E) * 0.1, torch.zeros(E, dtype=torch.int32, device="cuda")
    logits, choice = moe.route_tokens(h.cuda(), router.cuda(), E, K, corr.cuda(), counts, **how)
    assert (logits.double().cpu() - h.double() @ router.double().T).abs().max() < 2e-5
    rows, dest, w = moe.routed_experts(h.cuda(), choice, up.cuda(), down.cuda(), counts, moe.SILU_GATE)
    got = (rows[dest.long()].double() * w[:, :, None].double()).sum(1).cpu()
    z = logits.double().cpu()
    for t in range(T):
        want = 0
        for e, x in oracle.choose_experts(z[t], corr.double(), dict(top=K, scale=1.8, groups=dict(count=6, keep=3))):
            a = up[e].double() @ h[t].double()
            want = want + x * (down[e].double() @ (oracle.silu(a[:F]) * a[F:]))
        assert (got[t] - want).abs().max() < (1e-5 if dtype == "float32" else 3e-2) * want.abs().max().clamp_min(1), t


# ---------------------------------------------------------------------------------------------------- engine
@DTYPES
@pytest.mark.parametrize("which", ["uneven", "round"])
def test_portions_and_decoding_match_whole_sequences(which, dtype):
    c = lu.uneven_conf() if which == "uneven" else lu.round_conf()
    W = lu.weights(c, 5, dtype)
    eng = lu.make_engine(c, W, dtype, "cuda")
    for n, seed in ((1, 1), (2, 2), (150, 3), (260, 4)):
        seq = lu.tokens(n, c["vocab"], seed)
        want = oracle.forward(W, c, seq)
        for cuts in ([n], [1], [2], [64, 1], [15, 17, 1, 1, 100, 2]):
            if cuts == [1] and n > 200 or cuts == [2] and n < 200:
                continue
            lu.assert_close(lu.run_alone(eng, seq, cuts), want, dtype, (n, cuts))
    assert eng.get_load()["free_blocks"] == eng.num_blocks


@DTYPES
@pytest.mark.parametrize("block", [8, 64])
def test_mixed_batches_on_reused_pages_and_slots(dtype, block):
    c = lu.round_conf()
    W = lu.weights(c, 6, dtype)
    eng = lu.make_engine(c, W, dtype, "cuda", kv_block_size=block, num_kv_blocks=4 * 256 // block, max_model_len=256)
    seqs = [lu.tokens(n, c["vocab"], 20 + n) for n in (200, 31, 64, 1, 129, 65, 90, 17, 240)]
    for s, got in zip(seqs, lu.run_mixed(eng, seqs, [1, 1, 2, 3, 16, 63, 64, 65, 100], seed=7)):
        lu.assert_close(got, oracle.forward(W, c, s), dtype)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_the_batch_does_not_matter():
    """bf16 logits of one request alone and in a batch of others differ by rounding only."""
    c = lu.round_conf()
    W = lu.weights(c, 12, "bfloat16")
    eng = lu.make_engine(c, W, "bfloat16", "cuda", max_model_len=256)
    seqs = [lu.tokens(n, c["vocab"], 70 + n) for n in (120, 77, 33, 5)]
    for s, got in zip(seqs, lu.run_mixed(eng, seqs, [1, 2, 30, 64], seed=8)):
        lu.assert_close(got, lu.run_alone(eng, s, [len(s)]).double(), "bfloat16")


def test_true_32_bit_whatever_the_matrix_mode():
    """The 32-bit engine stays exact when the process allows TF32."""
    c = lu.round_conf()
    W = lu.weights(c, 8)
    eng = lu.make_engine(c, W, "float32", "cuda")
    seq = lu.tokens(70, c["vocab"], 9)
    torch.backends.cuda.matmul.allow_tf32 = True
    try:
        got = lu.run_alone(eng, seq, [40, 1])
    finally:
        torch.backends.cuda.matmul.allow_tf32 = False
    lu.assert_close(got, oracle.forward(W, c, seq))


@DTYPES
def test_greedy_generation_through_the_scheduler(dtype):
    """generate(): captured decode graphs, more requests than slots, prompts longer than a prefill step, samples that
    share a prompt - every token is the plain implementation's choice (or ties with it within rounding)."""
    c = lu.uneven_conf() if dtype == "float32" else lu.round_conf()
    W = lu.weights(c, 10, dtype)
    eng = lu.make_engine(c, W, dtype, "cuda", max_prefill_tokens=50, sync_interval=3, max_model_len=256)
    prompts = [lu.tokens(n, c["vocab"], 40 + n) for n in (1, 5, 33, 120, 64)]
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


def test_long_decoding_past_the_window():
    ly = [lu.attention(4, 2, 32, 64, 16, 0.17, 0.5, lu.dense(64)), lu.latent(4, 32, 8, 32, 64, 50, 0.15, lu.dense(64))]
    c = lu.conf(ly + [lu.again(ly, 1), lu.again(ly, 0)], 64, 128)
    W = lu.weights(c, 11, "bfloat16")
    eng = lu.make_engine(c, W, "bfloat16", "cuda", max_model_len=1024)
    seq = lu.tokens(400, c["vocab"], 12)
    lu.assert_close(lu.run_alone(eng, seq, [20] + [1] * 380), oracle.forward(W, c, seq), "bfloat16")


def _checkpoint(path, c, seed):
    from safetensors.torch import save_file
    W = lu.weights(c, seed, "bfloat16")
    save_file({k: v.contiguous() for k, v in W.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(c))
    return W


def test_command_line_generates_from_a_checkpoint_folder(tmp_path):
    from gcore_b200.entry import lm_infer
    c = lu.round_conf()
    W = _checkpoint(tmp_path, c, 13)
    prompts = [lu.tokens(n, c["vocab"], n) for n in (7, 20)]
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
    c = lu.uneven_conf()
    W = _checkpoint(tmp_path, c, 14)
    eng = trace_run.build_engine(str(tmp_path), "float32", 128, torch.device("cuda", 0))
    a, b = lu.tokens(40, c["vocab"], 1), lu.tokens(9, c["vocab"], 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[1:], want=[])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=b, want=[8]), dict(id="a", tokens=a[30:], want=[9])], end=["a", "c"])]
    said = []
    trace_run.replay(eng, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    la_, lb = oracle.forward(W, c, a), oracle.forward(W, c, b)
    for n, want in ((0, torch.stack([la_[0], la_[29], lb[0]])), (2, torch.stack([lb[8], la_[39]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"]).copy())
        lu.assert_close(got, want)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_serving_benchmark_runs_on_a_small_size():
    from gcore_b200.tools import serve_bench as sb
    from gcore_b200.tools import serve_bench_lobutar as sl
    s = dict(width=256, heads=4, kv=2, dim=32, vdim=96, lh=4, ldim=128, lrot=64, lv=128, rank=512, window=70, ff=512, experts=32,
             top=2, eff=192, groups=4, keep=2, streams=2, layers=4)
    for kind in ("lobutar", "grouped"):
        eng = sb.build(kind, s, 512, 4)
        assert sb.prefill_step(eng, 2, 130, 2) > 0 and sb.decode_step(eng, 4, 200, 2) > 0
        assert sl.decode_bytes(kind, s, eng, 4, 200) > 0
    table = sl.kernel_table(s, 2, 130, 4, 200)
    assert {r[0] for r in table} == {"prefill", "decode"} and all(r[2] > 0 for r in table)

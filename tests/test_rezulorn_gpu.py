"""Rezulorn on the GPU: every kernel alone against the plain implementation, then the engine - portions, mixed batches, freed
pages and slots, long decoding, generation - against whole sequences of the plain implementation."""
import json

import pytest
import torch

from gcore_b200.models.config import from_hf_config
from gcore_b200.models.plan_decoder import CheckpointTensors
from gcore_b200.models.plan_modules import RetentionMixer, ScoredAttentionMixer
from gcore_b200.ops import _lib
from gcore_b200.ops import conv_norm as cn
from gcore_b200.ops import head_prep as hp
from gcore_b200.ops import latent_attention as la
from gcore_b200.ops import matrix_memory as mm
from gcore_b200.rollout.engine import SamplingParams
from tests import rezulorn_util as ru
from tests.oracle import rezulorn as oracle

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
# portions: a fresh prompt, one behind a long context, two tokens across a page's and a tile's edge, more rows than one CTA of
# the prompt kernel takes; then single tokens
SEGS = [(0, 150), (333, 70), (63, 2), (127, 65), (5, 2), (40, 300), (500, 1), (0, 1), (64, 1), (255, 1), (31, 1)]


def _mixers(entry):
    return from_hf_config(ru.conf([entry], 8, 8)).layer_plan.layers[0].mixers


def _pad(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1]))


def _turned(rot):
    """Order of a head's dimensions in which the kernels keep it."""
    n = rot["dims"]
    return [i // 2 + (i % 2) * (n // 2) for i in range(n)]


def _attention_case(entry, left, m, dtype, bs, targets_of, check_rows):
    """One attention mixer over SEGS on shuffled pages.  Queries of ``check_rows`` single out one key each."""
    dt, eps = DT[dtype], 1e-4
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rows = ru.make_rows(SEGS, bs, sum((f + l + bs - 1) // bs for f, l in SEGS) + 5, 16)
    out_scale = 0.7
    mix = ScoredAttentionMixer(_mixers(entry)[0], 8, eps, dt, "cuda", out_scale)
    ly = mix.layout
    W = {n: torch.zeros(r, 8) for n, r in (("q", H * dim), ("k", G * dim), ("v", G * vdim))}
    W["o"] = torch.zeros(8, H * vdim)
    r1, r2, pb = torch.rand(H) + 0.3, torch.rand(H) * 2 + 0.02, torch.linspace(-9, -5, H)
    W.update(dict(pb=pb) if left else dict(r1=r1, r2=r2))
    mix.load(CheckpointTensors(W), "", torch.zeros(mix.columns, 8, device="cuda", dtype=dt),
             torch.zeros(8, mix.out_columns, device="cuda", dtype=dt))
    order = _turned(m["rot"]) + list(range(m["rot"]["dims"], dim)) if left else list(range(dim))
    ready = (lambda x, at: oracle.rms(oracle.rotate(x.double(), m["rot"], at), eps)) if left else (lambda x, at: x.double())
    tabs = rows.tables.cpu()
    where = lambda s, p: (tabs[s][p // bs].long() * bs + p % bs).cuda()
    cache = torch.full((int(rows.tables.max()) + 6, bs, ly.row), 3.0, dtype=dt, device="cuda")    # what earlier requests left
    flat = cache.view(-1, ly.row)
    lead = 16                                           # the mixer's columns need not start the row
    proj = torch.zeros(sum(l for _, l in SEGS), lead + mix.columns, dtype=dt, device="cuda")
    view, at, keep = proj[:, lead:], 0, []
    for s, (f, l) in enumerate(SEGS):
        n = f + l
        k0, v = torch.randn(n, G, dim).to(dt), torch.randn(n, G, vdim).to(dt)
        q = torch.randn(l, H, dim).to(dt)
        k = ready(k0, range(n)).to(dt).double()
        for r in check_rows(l):
            spots = targets_of(f + r, f)
            for h in range(H):
                key = k[spots[(h + r) % len(spots)], h // (H // G)]
                want = (key * 60 / key.pow(2).sum().sqrt())[None, None]
                q[r, h] = (oracle.rotate(want, m["rot"], [-(f + r)]) if left else want)[0, 0].to(dt)
        old = torch.cat([_pad(k[:f].to(dt)[..., order], ly.dim).flatten(1), _pad(v[:f], ly.vdim).flatten(1)], 1)
        flat[where(s, torch.arange(f))] = old.cuda()
        sl = view[at:at + l]
        sl[:, ly.q:ly.q + H * ly.dim] = _pad(q[..., order], ly.dim).flatten(1).cuda()
        sl[:, ly.k:ly.k + G * ly.dim] = _pad(k0[f:][..., order], ly.dim).flatten(1).cuda()
        sl[:, ly.v:ly.v + G * ly.vdim] = _pad(v[f:], ly.vdim).flatten(1).cuda()
        keep.append((s, at, f, l, ready(q, range(f, n)).to(dt).double(), k, v.double()))
        at += l
    out = torch.full((at, mix.out_columns + 8), 7.0, dtype=dt, device="cuda")
    mix(view, rows, cache, None, out[:, :mix.out_columns])
    _lib.check_device_errors()
    assert (out[:, mix.out_columns:] == 7).all()
    got = out[:, :mix.out_columns].view(at, H, ly.vdim).double().cpu()
    assert not got[..., vdim:].any()
    g = torch.arange(H) // (H // G)
    for s, at, f, l, q, k, v in keep:
        for r in sorted({0, 1, l // 2, l - 2, l - 1} & set(range(l))):
            i = f + r
            j = oracle.visible(i, m.get("mask"))
            sc = torch.einsum("hd,nhd->hn", q[r], k[j][:, g]) * m["scale"]
            if left:
                w = torch.sigmoid(sc + pb[:, None])
            else:
                d = torch.tensor([float(i - x) for x in j]).double()
                w = torch.softmax(sc - torch.stack([oracle.distance_penalty(d, a, b) for a, b in zip(r1.double(), r2.double())]), -1)
            want = torch.einsum("hn,nhv->hv", w, v[j][:, g]) * out_scale
            err = (got[at + r, :, :vdim] - want).abs().max() / want.abs().max().clamp_min(0.5)
            assert err < (2e-4 if dtype == "float32" else 4e-2), (f, l, r, float(err))
        stored = flat[where(s, torch.arange(f, f + l))].double().cpu()     # the new rows went to their slots, zero where padded
        ks, vs = stored[:, :ly.value_offset].view(l, G, ly.dim), stored[:, ly.value_offset:].view(l, G, ly.vdim)
        assert (ks[..., :dim] - k[f:][..., order]).abs().max() < (1e-5 if dtype == "float32" else 4e-2)
        assert torch.equal(vs[..., :vdim], v[f:]) and not ks[..., dim:].any() and not vs[..., vdim:].any()


# ---------------------------------------------------------------------------------------------- scored attention
@DTYPES
@pytest.mark.parametrize("H,G,dim,vdim,window,keep,bs", [
    (6, 2, 40, 72, 61, 3, 8), (16, 4, 64, 128, 64, 64, 64), (5, 5, 24, 40, 10, 1, 8), (12, 1, 128, 128, 128, 4, 32),
    (3, 3, 100, 60, 1, 0, 128), (20, 2, 56, 200, 33, 70, 16), (2, 1, 128, 256, 300, 0, 64), (40, 2, 32, 24, 65, 130, 16),
    (2, 2, 136, 48, 50, 6, 16), (4, 2, 20, 264, 17, 9, 16), (4, 2, 32, 64, 100, 40, 12), (4, 1, 128, 64, 4000, 5, 64)])
def test_distance_scored_attention_alone(H, G, dim, vdim, window, keep, bs, dtype):
    """Queries that single out the first key, the last kept and the next one, the keys just inside and just outside the
    window, the newest, the last of a page.  Sizes of every prompt and decode kernel, and of the general one."""
    torch.manual_seed(1)
    m = ru.attention(H, G, dim, vdim, window, keep, 0.4 * dim ** -0.5, 0)

    def spots(i, f):
        at = lambda p: min(max(p, 0), i)
        return [0, at(keep - 1), at(keep), at(i - window + 1), at(i - window), i, at(i - i % bs - 1), at(f - 1)]
    _attention_case(m, False, m["mixer"], dtype, bs, spots, lambda l: {0, 1, l // 2, l - 2, l - 1} & set(range(l)))


@DTYPES
@pytest.mark.parametrize("H,G,dim,vdim,rot,factor,bs", [
    (6, 2, 40, 72, 8, 3.0, 8), (16, 4, 64, 128, 64, None, 64), (5, 5, 24, 40, 10, 1.5, 8), (12, 1, 128, 128, 128, 2.0, 32),
    (3, 3, 100, 60, 100, None, 128), (20, 2, 56, 200, 6, 4.0, 16), (2, 1, 128, 256, 32, 2.0, 64), (40, 2, 32, 24, 32, None, 16),
    (2, 2, 136, 48, 16, 2.0, 16), (4, 2, 20, 264, 4, None, 16), (4, 2, 32, 64, 12, 8.0, 12), (4, 1, 128, 64, 64, 2.0, 64)])
def test_sigmoid_attention_alone(H, G, dim, vdim, rot, factor, bs, dtype):
    """Queries that single out the first key, the one in front of the portion, the last of a page, the newest."""
    torch.manual_seed(2)
    m = ru.gates(H, G, dim, vdim, ru.rotation(rot, 300.0, factor), 14.0 / dim)
    entry = ru.parallel(m, ru.retention(1, 8, 8, ru.rotation(2, 10.0), [0.5]), 1.0, 1.0, 0)

    def spots(i, f):
        at = lambda p: min(max(p, 0), i)
        return [0, i, at(f - 1), at(i - i % bs - 1), i // 2]
    _attention_case(entry, True, m, dtype, bs, spots, lambda l: {0, 1, l // 2, l - 2, l - 1} & set(range(l)))


@pytest.mark.parametrize("kind", ["distance", "sigmoid"])
@pytest.mark.parametrize("vdim", [64, 128, 232])
def test_decode_splits_agree(vdim, kind):
    """A long context cut into many splits = the same in one; kept positions far in front of the window."""
    torch.manual_seed(3)
    lib = _lib.kernels()
    entry = ru.attention(12, 4, 64, vdim, 1500, 200, 0.1, 0) if kind == "distance" else ru.parallel(
        ru.gates(12, 4, 64, vdim, ru.rotation(64, 500.0), 0.1), ru.retention(1, 8, 8, ru.rotation(2, 10.0), [0.5]), 1.0, 1.0, 0)
    mix = ScoredAttentionMixer(_mixers(entry)[0], 8, 1e-5, torch.bfloat16, "cuda", 0.5)
    for p in (mix.r1, mix.r2, mix.head_bias):
        if p is not None:
            p.uniform_(0.1, 0.9)
    ly = mix.layout
    rows = ru.make_rows([(5000, 1), (130, 1), (1499, 1), (1500, 1), (1600, 1)], 64, 160, 5)
    cache = torch.randn(161, 64, ly.row, device="cuda").bfloat16()
    proj = torch.randn(5, mix.columns, device="cuda").bfloat16()
    outs = []
    for target in (0, 1, 60):
        lib.gk_scored_set_target_ctas(target)
        out = torch.empty(5, mix.out_columns, dtype=torch.bfloat16, device="cuda")
        mix(proj.clone(), rows, cache.clone(), None, out)
        outs.append(out.float())
    lib.gk_scored_set_target_ctas(0)
    assert all((o - outs[0]).abs().max() < 2e-2 * outs[0].abs().max() for o in outs[1:]) and outs[0].abs().max() > 1e-2


def test_rotation_is_exact_far_out():
    """Positions up to a million, against float64; slowed pairs, then the norm, then without either."""
    rot = ru.rotation(16, 3000.0, 2.5)
    order, at = _turned(rot) + [16, 17, 18, 19], [0, 1, 77, 4095, 65537, 262143, 1000003]
    spec = _mixers(ru.parallel(ru.gates(1, 1, 20, 8, rot, 0.1), ru.retention(1, 8, 8, ru.rotation(2, 9.0), [0.5]), 1.0, 1.0, 0))[0].rot
    turns = la.rotation_turns(spec.frequencies()).cuda()
    rows = ru.make_rows([(0, 1)] * len(at), 16, 8, 8)
    rows.pos.copy_(torch.tensor(at))
    x = torch.randn(len(at), 3, 20)
    for kw, want in ((dict(turns=turns), oracle.rotate(x.double(), rot, at)),
                     (dict(turns=turns, unit_dim=20, eps=1e-3), oracle.rms(oracle.rotate(x.double(), rot, at), 1e-3)),
                     (dict(unit_dim=20, eps=1e-3), oracle.rms(x.double(), 1e-3)), (dict(), x.double())):
        proj = torch.full((len(at), 88), 5.0, device="cuda")
        proj[:, 8:80] = _pad(x[..., order], 24).flatten(1).cuda()
        hp.head_prep(proj, rows, 0, len(at), 8, 2, 56, 1, 24, **kw)
        got = proj[:, 8:80].view(-1, 3, 24).double().cpu()
        assert (got[..., :20] - want[..., order]).abs().max() < 3e-6 and not got[..., 20:].any()
        assert (proj[:, :8] == 5).all() and (proj[:, 80:] == 5).all()


def test_silu_columns():
    for dt in DT.values():
        x = 9 * torch.randn(4037, 4176, device="cuda").to(dt)
        y = x.clone()
        hp.silu_columns(y[3:], 16, 4152)
        want = oracle.silu(x[3:, 16:4168].double())
        assert ((y[3:, 16:4168].double() - want).abs() / want.abs().clamp_min(1)).max() < (1e-6 if dt == torch.float32 else 5e-3)
        y[3:, 16:4168] = x[3:, 16:4168]
        assert torch.equal(x, y)


def test_inactive_rows_leave_cache_and_state_alone():
    left = ru.gates(2, 1, 16, 24, ru.rotation(8, 50.0), 0.2)
    entry = ru.parallel(left, ru.retention(2, 16, 24, ru.rotation(8, 50.0), [0.5, 0.9]), 1.0, 1.0, 0)
    for dt in DT.values():
        rows = ru.make_rows([(9, 1), (20, 1)], 16, 8, 2)
        rows.slots[0], rows.ctx[0], rows.states[0] = -1, 0, -1
        for spec in (_mixers(ru.attention(2, 1, 16, 24, 7, 2, 0.2, 0))[0], _mixers(entry)[0]):
            mix = ScoredAttentionMixer(spec, 8, 1e-5, dt, "cuda")
            cache = torch.zeros(9, 16, *mix.cache_shape(), dtype=dt, device="cuda")
            out = torch.ones(2, mix.out_columns, dtype=dt, device="cuda")
            mix(torch.ones(2, mix.columns, dtype=dt, device="cuda"), rows, cache, None, out)
            assert not out[0].any() and out[1].any() and (cache.view(-1, mix.layout.row).abs().sum(-1) > 0).sum() == 1
        for spec in (_mixers(entry)[1], _mixers(ru.lightning(2, 16, 24, [0.5, 0.9], 0))[0]):
            mix = RetentionMixer(spec, 8, 1e-5, dt, "cuda")
            st = mix.new_state(3, "cuda")
            out = torch.ones(2, mix.out_columns, dtype=dt, device="cuda")
            mix(torch.ones(2, mix.columns, dtype=dt, device="cuda"), rows, None, st, out)
            assert not out[0].any()
            assert [bool(st.S[i].any()) for i in range(3)] == [i == int(rows.states[1]) for i in range(3)]


# ---------------------------------------------------------------------------------------------- memories
@DTYPES
@pytest.mark.parametrize("kind", ["rotated", "activated"])
@pytest.mark.parametrize("heads,dim,vdim,rot", [(3, 20, 36, 14), (2, 64, 64, 64), (4, 128, 128, 32), (2, 200, 72, 200),
                                                (1, 16, 520, 4), (2, 300, 24, 300)])
def test_memories_alone(heads, dim, vdim, rot, kind, dtype):
    """Portions that start fresh and from a state, of a few tokens and of several chunks, beside single tokens: outputs and
    the state left behind, with decays from nearly nothing to one."""
    torch.manual_seed(4)
    dt, eps, scale = DT[dtype], 1e-4, 1.3
    segs = [(0, 290), (700, 130), (3, 2), (128, 9), (0, 5), (40, 1), (0, 1), (17, 1)]
    decay = [0.999, 0.6, 1.0, 0.02][:heads]
    r = ru.rotation(rot, 200.0, 2.0)
    entry = ru.parallel(ru.gates(1, 1, 8, 8, ru.rotation(2, 9.0), 0.1), ru.retention(heads, dim, vdim, r, decay), 1.0, 1.0, 0)
    spec = _mixers(entry)[1] if kind == "rotated" else _mixers(ru.lightning(heads, dim, vdim, decay, 0))[0]
    mix = RetentionMixer(spec, 8, eps, dt, "cuda", scale)
    order = _turned(r) + list(range(rot, dim)) if kind == "rotated" else list(range(dim))
    if mix.gain is not None:
        gain = torch.rand(heads, vdim) + 0.5
        mix.gain.view(heads, -1)[:, :vdim] = gain.cuda()
    rows = ru.make_rows(segs, 16, 200, 12)
    st = mix.new_state(12, "cuda")
    st.S.fill_(100.0)                                   # what earlier requests left
    T = sum(l for _, l in segs)
    proj = torch.zeros(T, mix.columns, dtype=dt, device="cuda")
    q, k, v, g = (torch.randn(T, heads, d).to(dt) for d in (dim, dim, vdim, vdim))
    for x, at, pad in ((q[..., order], mix.at[0], mix.dim), (k[..., order], mix.at[1], mix.dim), (v, mix.at[2], mix.vdim),
                       (g, mix.at[3], mix.vdim)):
        proj[:, at:at + heads * pad] = _pad(x, pad).flatten(1).cuda()
    S0 = torch.randn(len(segs), heads, dim, vdim)
    for s, (f, l) in enumerate(segs):
        if f:
            st.S[rows.states[s].long()] = 0
            st.S[rows.states[s].long(), :, :dim, :vdim] = S0[s][:, order].cuda()
    out = torch.full((T, mix.out_columns + 8), 7.0, dtype=dt, device="cuda")
    mix(proj, rows, None, st, out[:, :mix.out_columns])
    _lib.check_device_errors()
    assert (out[:, mix.out_columns:] == 7).all()
    got, at = out[:, :mix.out_columns].view(T, heads, mix.vdim).double().cpu(), 0
    for s, (f, l) in enumerate(segs):
        sl, pos = slice(at, at + l), range(f, f + l)
        qq, kk, vv = q[sl].double(), k[sl].double(), v[sl].double()
        if kind == "rotated":
            qq, kk = oracle.rotate(qq, r, pos), oracle.rotate(kk, r, pos)
        else:
            qq, kk, vv = oracle.silu(qq), oracle.silu(kk), oracle.silu(vv)
        if dtype == "bfloat16" and l > 1:               # prepared in place
            qq, kk, vv = (x.to(dt).double() for x in (qq, kk, vv))
        S = S0[s].double() if f else torch.zeros(heads, dim, vdim).double()
        o = torch.zeros(l, heads, vdim).double()
        for t in range(l):
            S = torch.tensor(decay).double()[:, None, None] * S + kk[t][:, :, None] * vv[t][:, None]
            o[t] = torch.einsum("hdv,hd->hv", S, qq[t]) * spec.product_scale()
        gate = g[sl].double()
        want = oracle.rms(o, eps) * oracle.silu(gate) if kind == "rotated" else \
            oracle.rms(o.flatten(1), eps).view(o.shape) * gain * torch.sigmoid(gate)
        err = (got[sl, :, :vdim] - want * scale).abs().max()
        assert err < (1e-3 if dtype == "float32" else 6e-2), (f, l, float(err))
        left = st.S[rows.states[s].long()].double().cpu()
        assert (left[:, :dim, :vdim] - S[:, order]).abs().max() < 2e-4 * S.abs().max(), (f, l)
        at += l
    assert not got[..., vdim:].any()


# ---------------------------------------------------------------------------------------------- residual steps
@DTYPES
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 13])
@pytest.mark.parametrize("width,pad", [(44, 48), (600, 600), (1500, 1504), (4096, 4096), (12000, 12000)])
def test_convolved_norm_alone(width, pad, taps, dtype):
    """Portions shorter than the convolution and longer than a strip, fresh and from a ring, beside single tokens: the
    residual, the convolved norm, and the ring left behind."""
    torch.manual_seed(5)
    dt, eps, V, mult = DT[dtype], 1e-3, 31, 0.6
    segs = [(0, 37), (50, 61), (3, 2), (128, 5), (1, 3), (40, 1), (0, 1), (2, 1)]
    T = sum(l for _, l in segs)
    rows = ru.make_rows(segs, 16, 60, 12)
    rows.tokens = torch.randint(0, V, (T,), device="cuda")
    stored = cn.stored_taps(taps)
    c = lambda t: _pad(t, pad).contiguous().cuda()
    w, gain = torch.randn(width, taps) * 0.5, torch.rand(width) + 0.5
    tp = torch.zeros(stored, width)
    tp[stored - taps:] = w.t()
    tp[-1] += 1
    embed, y, x0 = torch.randn(V, width).to(dt) + 3, torch.randn(T, width).to(dt), torch.randn(T, width) - 2
    past = torch.randn(len(segs), 200, width)           # normed inputs of earlier steps, by position
    tol = 5e-5 if dtype == "float32" else 6e-2
    spec = cn.NormSpec(width, eps)
    for source in ("embed", "add"):
        ring = torch.full((12, stored - 1, pad), 50.0, device="cuda")
        for s, (f, l) in enumerate(segs):
            for p in range(max(0, f - stored + 1), f):
                ring[rows.states[s].long(), p % (stored - 1)] = c(past[s, p])
        before = ring.clone()
        if source == "embed":
            x, h = cn.conv_embed_rows(rows, c(embed), c(gain), c(tp), ring, spec)
            res = embed[rows.tokens.cpu()].double()
        else:
            x, h = cn.conv_add_sublayer(c(x0), c(y), mult, spec, c(gain), rows, c(tp), ring)
            res = x0.double() + mult * y.double()
        assert (x[:, :width].double().cpu() - res).abs().max() < 1e-5 and not x[:, width:].any() and not h[:, width:].any()
        n, at, used = oracle.layer_norm(res, gain.double(), eps), 0, set()
        for s, (f, l) in enumerate(segs):
            seq = torch.cat([past[s, :f].double(), n[at:at + l]])
            want = oracle.input_conv(seq[max(0, f - taps + 1):], w.double())[-l:]
            assert (h[at:at + l, :width].double().cpu() - want).abs().max() < tol * want.abs().max().clamp_min(1), (source, f, l)
            slot = int(rows.states[s])
            used.add(slot)
            for p in range(max(0, f + l - stored + 1), f + l):
                assert (ring[slot, p % (stored - 1), :width].double().cpu() - seq[p]).abs().max() < 2e-5 * seq[p].abs().max().clamp_min(1)
            at += l
        rest = [i for i in range(12) if i not in used]
        assert torch.equal(ring[rest], before[rest])
    x, h = cn.conv_add_sublayer(c(x0), c(y), mult, spec, c(gain), keep=False)
    want = oracle.layer_norm(x0.double() + mult * y.double(), gain.double(), eps)
    assert x is None and (h[:, :width].double().cpu() - want).abs().max() < tol
    x, h = cn.conv_add_sublayer(c(x0), c(y), mult, spec)
    pick = torch.tensor([5, 0, 60], device="cuda")
    got = cn.conv_norm_rows(x, c(gain), spec, dt, pick)
    assert h is None and (got[:, :width].double().cpu() - want[[5, 0, 60]]).abs().max() < tol
    bare = cn.conv_norm_rows(x, c(gain), cn.NormSpec(width, eps, center=False), dt)
    assert (bare[:, :width].double().cpu() - oracle.rms(x0.double() + mult * y.double(), eps) * gain).abs().max() < tol


def test_strips_of_every_length_agree():
    """However a long portion is cut, neighbouring strips see the same rows; lengths around the strips' edges."""
    torch.manual_seed(6)
    lib, H = _lib.kernels(), 256
    for stored in (2, 3, 4):
        segs = [(3, n) for n in (1200, 29, 30, 5, 6, 13, 2)]
        T = sum(l for _, l in segs)
        rows = ru.make_rows(segs, 16, 200, 8)
        x, y, gain, taps = (torch.randn(*s, device="cuda") for s in ((T, H), (T, H), (H,), (stored, H)))
        start, outs = torch.randn(8, stored - 1, H, device="cuda"), []
        for n in (1, 2, 3, 4, 0):
            lib.gk_conv_norm_set_rounds(n)
            ring = start.clone()
            outs.append((*cn.conv_add_sublayer(x, y, 0.7, cn.NormSpec(H, 1e-5), gain, rows, taps, ring), ring))
        assert all(torch.equal(a, b) for o in outs[1:] for a, b in zip(o, outs[0]))


# ---------------------------------------------------------------------------------------------------- engine
@DTYPES
@pytest.mark.parametrize("which", ["uneven", "round"])
def test_portions_and_decoding_match_whole_sequences(which, dtype):
    c = ru.uneven_conf() if which == "uneven" else ru.round_conf()
    W = oracle.random_weights(c, 5)
    eng = ru.make_engine(c, W, dtype, "cuda")
    for n, seed in ((1, 1), (2, 2), (150, 3), (290, 4)):
        seq = ru.tokens(n, c["vocab"], seed)
        want = ru.forward(W, c, seq)
        for cuts in ([n], [1], [2], [64, 1], [15, 17, 1, 1, 100, 2]):
            if cuts == [1] and n > 200 or cuts == [2] and n < 200:
                continue
            ru.assert_close(ru.run_alone(eng, seq, cuts), want, dtype, (n, cuts))
    assert eng.get_load()["free_blocks"] == eng.num_blocks


@DTYPES
@pytest.mark.parametrize("block", [8, 64])
def test_mixed_batches_on_reused_pages_and_slots(dtype, block):
    c = ru.round_conf(taps=4)
    W = oracle.random_weights(c, 6)
    eng = ru.make_engine(c, W, dtype, "cuda", kv_block_size=block, num_kv_blocks=4 * 256 // block, max_model_len=256)
    seqs = [ru.tokens(n, c["vocab"], 20 + n) for n in (200, 31, 64, 1, 129, 65, 90, 17, 240)]
    for s, got in zip(seqs, ru.run_mixed(eng, seqs, [1, 1, 2, 3, 16, 63, 64, 65, 100], seed=7)):
        ru.assert_close(got, ru.forward(W, c, s), dtype)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_the_batch_does_not_matter():
    """bf16 logits of one request alone and in a batch of others differ by rounding only."""
    c = ru.round_conf()
    W = oracle.random_weights(c, 12)
    eng = ru.make_engine(c, W, "bfloat16", "cuda", max_model_len=256)
    seqs = [ru.tokens(n, c["vocab"], 70 + n) for n in (120, 77, 33, 5)]
    for s, got in zip(seqs, ru.run_mixed(eng, seqs, [1, 2, 30, 64], seed=8)):
        ru.assert_close(got, ru.run_alone(eng, s, [len(s)]).double(), "bfloat16")


def test_true_32_bit_whatever_the_matrix_mode():
    """The 32-bit engine stays exact when the process allows TF32."""
    c = ru.round_conf()
    W = oracle.random_weights(c, 8)
    eng = ru.make_engine(c, W, "float32", "cuda")
    seq = ru.tokens(70, c["vocab"], 9)
    torch.backends.cuda.matmul.allow_tf32 = True
    try:
        got = ru.run_alone(eng, seq, [40, 1])
    finally:
        torch.backends.cuda.matmul.allow_tf32 = False
    ru.assert_close(got, ru.forward(W, c, seq))


@DTYPES
def test_greedy_generation_through_the_scheduler(dtype):
    """generate(): captured decode graphs, more requests than slots, prompts longer than a prefill step, samples that
    share a prompt - every token is the plain implementation's choice (or ties with it within rounding)."""
    c = ru.uneven_conf() if dtype == "float32" else ru.round_conf()
    W = oracle.random_weights(c, 10)
    eng = ru.make_engine(c, W, dtype, "cuda", max_prefill_tokens=50, sync_interval=3, max_model_len=256)
    prompts = [ru.tokens(n, c["vocab"], 40 + n) for n in (1, 5, 33, 120, 64)]
    reqs = eng.generate(prompts, SamplingParams(max_new_tokens=40, greedy=True), n=2)
    assert eng.stats["graph_replays"] > 0
    for k, r in enumerate(reqs):
        assert len(r.out_tokens) == 40
        if dtype == "float32":
            assert r.out_tokens == reqs[k // 2 * 2].out_tokens
        if k % 2 == 0:
            lg = ru.forward(W, c, r.prompt + r.out_tokens)[len(r.prompt) - 1:-1]
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert gap.max() < (1e-4 if dtype == "float32" else 0.25) * lg.std(), float(gap.max())
            lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(r.out_tokens)[:, None])[:, 0]
            assert (lp - torch.tensor(r.out_logprobs)).abs().max() < (1e-3 if dtype == "float32" else 0.5) * lg.std().clamp_min(1)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_long_decoding_past_the_window():
    ly = [ru.attention(4, 2, 32, 64, 50, 6, 0.17, 64), ru.lightning(2, 32, 32, [0.99, 0.9], 64),
          ru.parallel(ru.gates(4, 2, 32, 32, ru.rotation(32, 100.0), 0.3), ru.retention(2, 32, 32, ru.rotation(16, 100.0), [0.9, 0.999]),
                      0.5, 1.0, 64)]
    c = ru.conf(ly, 64, 128, taps=2)
    W = oracle.random_weights(c, 11)
    eng = ru.make_engine(c, W, "bfloat16", "cuda", max_model_len=1024)
    seq = ru.tokens(400, c["vocab"], 12)
    ru.assert_close(ru.run_alone(eng, seq, [20] + [1] * 380), ru.forward(W, c, seq), "bfloat16")


def _checkpoint(path, c, seed):
    from safetensors.torch import save_file
    W = oracle.random_weights(c, seed)
    save_file({k: v.contiguous() for k, v in W.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(c))
    return W


def test_command_line_generates_from_a_checkpoint_folder(tmp_path):
    from gcore_b200.entry import lm_infer
    c = ru.round_conf()
    W = _checkpoint(tmp_path, c, 13)
    prompts = [ru.tokens(n, c["vocab"], n) for n in (7, 20)]
    (tmp_path / "p.jsonl").write_text("".join(json.dumps({"prompt_token_ids": p}) + "\n" for p in prompts))
    out = tmp_path / "o.jsonl"
    lm_infer.main([f"checkpoint.load_ckpt_path={tmp_path}", f"+task.infer.prompts={tmp_path}/p.jsonl",
                   f"+task.infer.out={out}", "+task.infer.greedy=true"])
    got = [json.loads(l) for l in out.read_text().splitlines()]
    assert [g["prompt_length"] for g in got] == [7, 20]
    for g, p in zip(got, prompts):
        assert len(g["tokens"]) == len(p) + 128 and g["tokens"][:len(p)] == p
        lg = ru.forward(W, c, g["tokens"][:len(p) + 20])[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(g["tokens"][len(p):len(p) + 20])[:, None])[:, 0]
        assert gap.max() < 0.25 * lg.std()


def test_trace_replay_through_the_executable_entry(tmp_path):
    import numpy as np

    from gcore_b200.entry import trace_run
    c = ru.uneven_conf()
    W = _checkpoint(tmp_path, c, 14)
    eng = trace_run.build_engine(str(tmp_path), "float32", 128, torch.device("cuda", 0))
    a, b = ru.tokens(40, c["vocab"], 1), ru.tokens(9, c["vocab"], 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29]), dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[1:], want=[])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=b, want=[8]), dict(id="a", tokens=a[30:], want=[9])], end=["a", "c"])]
    said = []
    trace_run.replay(eng, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    fa, fb = ru.forward(W, c, a), ru.forward(W, c, b)
    for n, want in ((0, torch.stack([fa[0], fa[29], fb[0]])), (2, torch.stack([fb[8], fa[39]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"]).copy())
        ru.assert_close(got, want)
    assert eng.get_load()["free_blocks"] == eng.num_blocks


def test_serving_benchmark_runs_on_a_small_size():
    from gcore_b200.tools import serve_bench as sb
    from gcore_b200.tools import serve_bench_rezulorn as sr
    s = dict(width=256, heads=4, kv=2, dim=64, window=70, keep=5, rh=2, rk=64, rv=64, lh=2, lk=64, lv=64, ff=768, nff=512, layers=3,
             taps=3, mh=2, mk=64, mv=64)
    for kind in ("rezulorn", "nafitar", "mixed"):
        eng = sb.build(kind, s, 512, 4)
        assert sb.prefill_step(eng, 2, 130, 2) > 0 and sb.decode_step(eng, 4, 200, 2) > 0
        assert sr.decode_bytes(kind, s, eng, 4, 200) > 0
    table = sr.kernel_table(s, 2, 130, 4, 200)
    assert {r[0] for r in table} == {"prefill", "decode"} and all(r[2] > 0 for r in table)

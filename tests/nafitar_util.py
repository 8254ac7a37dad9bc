"""Shared pieces of the Nafitar tests: small configurations, engines on them, schedules of portions."""
import random
from dataclasses import replace

import torch

from gcore_b200.models.config import from_hf_config
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.rollout.engine import InferEngine, RolloutWeights


def layer_conf(heads, kv_heads, dim, window, scale, mem_heads, mem_dim, mem_vdim, cap, ff):
    return dict(type="parallel", mlp=None if ff is None else dict(ff=ff, kind="dense"), mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=window), scale=scale),
        right=dict(heads=mem_heads, dim=mem_dim, vdim=mem_vdim, gate_cap=cap)))


def conf(layers, width, vocab, loop=None, positions=512, eps=1e-5):
    c = dict(architecture="Nafitar", layers=layers, max_positions=positions, norm=dict(eps=eps), vocab=vocab, width=width)
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def uneven_conf(positions=512):
    """Layers that share no size, odd widths everywhere, one layer without a feed-forward, a loop in the middle."""
    return conf([layer_conf(6, 3, 20, 37, 0.3, 3, 12, 20, 5.0, 36), layer_conf(4, 1, 16, 5, 0.2, 2, 8, 24, 9.0, None),
                 layer_conf(2, 2, 24, 2, 0.25, 1, 40, 70, 3.0, 44)], width=44, vocab=75, loop=(1, 3, 3), positions=positions)


def round_conf(window=70, loop=(0, 1, 2), positions=1024):
    """Two equal layers with sizes the tensor-core kernels take without padding."""
    return conf([layer_conf(8, 2, 128, window, 0.09, 4, 64, 128, 12.0, 192)] * 2, width=192, vocab=320, loop=loop,
                positions=positions)


def make_engine(c, W, dtype="float32", device="cpu", **kw):
    cfg = replace(from_hf_config(c), dtype=dtype)
    model = build_decoder(cfg, device).load_tensors(W)
    kw = {**dict(max_running_requests=4, max_model_len=min(c["max_positions"], 512), kv_block_size=16,
                 use_cuda_graph=device != "cpu"), **kw}
    return InferEngine(cfg, RolloutWeights.from_model(model), device=torch.device(device), **kw)


def tokens(n, vocab, seed):
    g = random.Random(seed)
    return [g.randrange(vocab) for _ in range(n)]


def run_alone(engine, seq, cuts):
    """Logits of every position of one request whose tokens come in portions of ``cuts`` (repeated as needed)."""
    rid, at, out, i = engine.open_request(), 0, [], 0
    while at < len(seq):
        n = min(cuts[i % len(cuts)], len(seq) - at)
        out.append(engine.step([(rid, seq[at:at + n])], [list(range(n))]).cpu())
        at, i = at + n, i + 1
    engine.close_request(rid)
    return torch.cat(out)


def run_mixed(engine, seqs, sizes, seed, live_limit=4, skip=0.25):
    """Logits of every position of several requests that enter, pause and leave at random, cut into random portions."""
    g = random.Random(seed)
    todo, live, out = list(range(len(seqs))), {}, {i: [] for i in range(len(seqs))}
    while todo or live:
        while todo and len(live) < live_limit:
            live[todo.pop(0)] = [engine.open_request(), 0]
        entries, want, ids = [], [], []
        for i, (rid, at) in live.items():
            if g.random() < skip:
                continue
            n = min(g.choice(sizes), len(seqs[i]) - at)
            entries.append((rid, seqs[i][at:at + n]))
            want.append(list(range(n)))
            ids.append(i)
        if not entries:
            continue
        lg, k = engine.step(entries, want).cpu(), 0
        for i, w in zip(ids, want):
            out[i].append(lg[k:k + len(w)])
            k += len(w)
            live[i][1] += len(w)
            if live[i][1] == len(seqs[i]):
                engine.close_request(live.pop(i)[0])
    return [torch.cat(out[i]) for i in range(len(seqs))]


def rms_error(got, want):
    """Error of every position: mean over the vocabulary taken off, relative to the spread of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()


def assert_close(got, want, dtype="float32", what=None):
    """Rounding-sized errors only.  In bf16 a few positions are ill-conditioned (a memory read-out that nearly cancels is
    blown up by its norm), so nine in ten must be close and none far."""
    e = rms_error(got, want)
    worst, bulk = (2e-4, 2e-5) if dtype == "float32" else (0.8, 5e-2)
    assert e.max() < worst and e.quantile(0.9) < bulk, (what, float(e.max()), float(e.quantile(0.9)), int(e.argmax()))

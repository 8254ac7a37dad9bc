"""Shared pieces of the layer-plan decoders' tests: engines on small configurations, schedules of portions, comparisons."""
import random
from dataclasses import replace

import torch

from gcore_b200.models.config import from_hf_config
from gcore_b200.models.plan_decoder import build_decoder
from gcore_b200.ops.rows import PortionContexts, StepRows, portion_contexts
from gcore_b200.rollout.engine import InferEngine, RolloutWeights


def make_rows(segments, block_size, n_blocks, n_slots, seed=0, device="cuda", windows=(0,)):
    """StepRows of ``segments`` = [(first position, length)] on shuffled cache blocks and state slots; portions (length
    > 1) must come first.  ``windows``: the attention windows whose contexts the rows carry."""
    g = torch.Generator().manual_seed(seed)
    perm = torch.randperm(n_blocks, generator=g).tolist()
    mb = max((f + l + block_size - 1) // block_size for f, l in segments)
    tab = torch.zeros(len(segments), mb, dtype=torch.int32)
    for i, (f, l) in enumerate(segments):
        for b in range((f + l + block_size - 1) // block_size):
            tab[i, b] = perm.pop()
    lens = [l for _, l in segments]
    n_port = sum(l > 1 for l in lens)
    assert all(l > 1 for l in lens[:n_port])
    seq = torch.repeat_interleave(torch.arange(len(segments), dtype=torch.int32), torch.tensor(lens))
    pos = torch.cat([torch.arange(f, f + l, dtype=torch.int32) for f, l in segments])
    slots = tab[seq.long(), (pos // block_size).long()] * block_size + pos % block_size
    cu = torch.tensor([sum(lens[:i]) for i in range(n_port + 1)], dtype=torch.int32)
    states = torch.randperm(n_slots, generator=g)[:len(segments)].to(torch.int32)
    first = torch.tensor([f for f, _ in segments], dtype=torch.int32)
    d = lambda t: t.to(device)
    contexts = {}
    for w in windows:
        start, off, n, before = portion_contexts([f for f, _ in segments[:n_port]], lens[:n_port], w)
        contexts[w] = PortionContexts(cu=d(off), start=d(start) if w else None, rows=n, max_before=before)
    return StepRows(tokens=torch.zeros(pos.numel(), dtype=torch.int64, device=device), pos=d(pos), slots=d(slots.int()),
                    tables=d(tab), states=d(states), first_pos=d(first), cu=d(cu), ctx=d((first + 1)[n_port:].contiguous()),
                    row_seq=d(seq), n_portions=n_port, portion_rows=int(cu[-1]), max_portion=max(lens[:n_port], default=0),
                    max_ctx=max((f + 1 for f, l in segments if l == 1), default=1), contexts=contexts)


def make_engine(c, W, dtype="float32", device="cpu", **kw):
    cfg = replace(from_hf_config(c), dtype=dtype)
    model = build_decoder(cfg, device).load_tensors(W)
    kw = {**dict(max_running_requests=4, max_model_len=min(c.get("max_positions", 512), 512), kv_block_size=16,
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

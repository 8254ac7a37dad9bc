"""Serving throughput of layer-plan decoders beside the closest uniform model at equal size (``bench.py --serve``).

For a few real-model layer sizes (random weights) it times, on the device, a prefill step and a captured decode step of an
engine of the design and of the closest uniform model - for Nafitar a dense grouped-query decoder with the same width,
heads, window, feed-forward and layer count, for Kedesun and Lobutar a latent-attention decoder with experts
(``serve_bench_kedesun.py``, ``serve_bench_lobutar.py``), for Rezulorn both Nafitar and a dense decoder
(``serve_bench_rezulorn.py``) - and then every kernel the design added beside the like kernel of that model: time, the time its
bytes or FLOPs would take at the measured peaks, and the ratio of the two.  Inputs of every timed launch rotate over buffers larger than L2."""
from __future__ import annotations

import json
import math
import os

import torch

from ..models.config import ModelConfig, from_hf_config
from ..models.gpt import GPTModel
from ..models.plan_decoder import build_decoder
from ..ops import _lib, attention, fused, sandwich
from ..ops import matrix_memory as mm
from ..ops import window_attention as wa
from ..ops.rows import PortionContexts, StepRows
from ..rollout.engine import InferEngine, RolloutWeights, SamplingParams

SIZES = {
    # name: width, heads, kv heads, head dim, window, memory heads, key dim, value dim, feed-forward, layers
    "2k": dict(width=2048, heads=16, kv=4, dim=128, window=1024, mh=8, mk=128, mv=256, ff=5632, layers=12),
    "4k": dict(width=4096, heads=32, kv=8, dim=128, window=2048, mh=16, mk=128, mv=256, ff=11008, layers=8),
    "3k-wide-keys": dict(width=3072, heads=24, kv=8, dim=128, window=1024, mh=6, mk=256, mv=512, ff=8192, layers=8),
}
VOCAB = 32768


def peaks():
    path = os.path.join(os.path.dirname(__file__), "..", "..", "MEASURED_PEAKS.json")
    try:
        p = json.load(open(path))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    except Exception:  # noqa: BLE001
        return 6.65e12, 1.59e15, "fallback"


def nafitar_conf(s, positions):
    layer = dict(type="parallel", mlp=dict(ff=s["ff"], kind="dense"), mixer=dict(
        left=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["dim"], mask=dict(size=s["window"]),
                  scale=s["dim"] ** -0.5),
        right=dict(heads=s["mh"], dim=s["mk"], vdim=s["mv"], gate_cap=15.0)))
    return dict(architecture="Nafitar", layers=[layer] * s["layers"], max_positions=positions, norm=dict(eps=1e-6),
                vocab=VOCAB, width=s["width"])


def dense_config(s):
    return ModelConfig(arch="llama", num_layers=s["layers"], hidden_size=s["width"], num_attention_heads=s["heads"],
                       num_kv_heads=s["kv"], head_dim=s["dim"], ffn_hidden_size=s["ff"], vocab_size=VOCAB, qkv_bias=True,
                       sliding_window=s["window"])


def build(kind, s, positions, requests, block=64):
    """Engine of a layer-plan design (``nafitar``, ``kedesun``, ``lobutar``, ``rezulorn``) or of the uniform model it is compared
    with (``dense``, ``latent``: Kedesun's, ``grouped``: Lobutar's, ``mixed``: Rezulorn's dense one)."""
    from . import serve_bench_kedesun as sk, serve_bench_lobutar as sl, serve_bench_rezulorn as sr
    dev = torch.device("cuda")
    plans = {"nafitar": lambda: nafitar_conf(sr.like_sizes(s) if "nff" in s else s, positions), "kedesun": lambda: sk.conf(s),
             "lobutar": lambda: sl.conf(s), "rezulorn": lambda: sr.conf(s)}
    if kind in plans:
        cfg = from_hf_config(plans[kind]())
        model = build_decoder(cfg, dev).randomize()
    else:
        cfg = {"dense": dense_config, "latent": sk.latent_config, "grouped": sl.latent_config, "mixed": sr.dense_config}[kind](s)
        model = GPTModel(cfg, recompute="none", device=dev)
    eng = InferEngine(cfg, RolloutWeights.from_model(model), max_running_requests=requests, max_model_len=positions,
                      kv_block_size=block, max_prefill_tokens=1 << 20, device=dev)
    eng.wake_up()
    return eng


def event_ms(fn, iters, warm=3):
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def prefill_step(eng, prompts, length, iters):
    """ms of one prefill step over ``prompts`` prompts of ``length`` tokens."""
    dev = eng.device
    toks = torch.randint(0, VOCAB, (prompts, length)).tolist()
    if eng.plan is not None:
        rids = [eng.open_request() for _ in range(prompts)]
        for r in rids:
            assert eng.sched.reserve(r, length) == 0
        rows, _ = eng._step_rows([(r, 0, t) for r, t in zip(rids, toks)])
        last = rows.cu[1:].long() - 1

        def run():
            with torch.no_grad():
                eng.plan.final_rows(eng.plan(rows, eng.k_cache, eng.memory, final=False), last)
        ms = event_ms(run, iters)
        for r in rids:
            eng.close_request(r)
        return ms
    t = torch.tensor(toks, device=dev).reshape(-1)
    pos = torch.arange(length, dtype=torch.int32, device=dev).repeat(prompts)
    cu = torch.arange(prompts + 1, dtype=torch.int32, device=dev) * length
    per = (length + eng.bs - 1) // eng.bs * eng.bs
    slots = (torch.arange(prompts, device=dev)[:, None] * per + torch.arange(length, device=dev)).reshape(-1).int()
    return event_ms(lambda: eng._prefill(t, pos, cu, length, slots), iters)


def decode_state(eng, B, ctx):
    st = eng._new_state(B, SamplingParams(greedy=True))
    nb = (ctx + 128 + eng.bs - 1) // eng.bs
    assert B * nb <= eng.num_blocks
    st["active"].fill_(True)
    st["pos"].fill_(ctx)
    st["limit"].fill_(ctx + 128)
    st["state"].copy_(torch.arange(B))
    st["block_table"][:, :nb] = torch.arange(B * nb, dtype=torch.int32, device=eng.device).view(B, nb)
    return st


def decode_step(eng, B, ctx, iters):
    st = decode_state(eng, B, ctx)

    def run():
        st["pos"].fill_(ctx)
        eng._run_decode(st)
    ms = event_ms(run, iters)
    eng._graphs.clear()
    return ms


def model_bytes(eng):
    return sum(t.numel() * t.element_size() for t in eng.w.tensors()) - eng.w.embed.numel() * eng.w.embed.element_size()


def decode_bytes(kind, s, eng, B, ctx):
    """HBM bytes one decode step has to move: weights once, the visible cache, the recurrent state in and out."""
    span = min(ctx + 1, s["window"])
    cache = B * span * s["kv"] * s["dim"] * 2 * s["layers"] * (1 if kind == "nafitar" else 2)
    state = 2 * 4 * B * s["mh"] * s["mk"] * s["mv"] * s["layers"] if kind == "nafitar" else 0
    return model_bytes(eng) + cache + state


# ------------------------------------------------------------------------------------------------------ kernels alone
def graph_us(fns, replays=20):
    """Microseconds per launch of ``fns`` (same kernel on rotating inputs), captured into one graph."""
    for f in fns:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in fns:
            f()
    return event_ms(g.replay, replays) * 1e3 / len(fns)


def _rows(prompts, length, ctx, B, bs, dev, windows=(0,)):
    """Rows of ``prompts`` whole prompts, or (``prompts`` = 0) of B single tokens at context ``ctx``."""
    if prompts:
        n, T = prompts, prompts * length
        nb = (length + bs - 1) // bs
        pos = torch.arange(length, dtype=torch.int32, device=dev).repeat(n)
        seq = torch.arange(n, dtype=torch.int32, device=dev).repeat_interleave(length)
        first = torch.zeros(n, dtype=torch.int32, device=dev)
        cu = torch.arange(n + 1, dtype=torch.int32, device=dev) * length
        ctxs = torch.zeros(0, dtype=torch.int32, device=dev)
    else:
        n, T, nb = B, B, (ctx + bs) // bs
        pos = torch.full((n,), ctx, dtype=torch.int32, device=dev)
        seq = torch.arange(n, dtype=torch.int32, device=dev)
        first, cu, ctxs = pos, None, pos + 1
    contexts = {w: PortionContexts(cu=cu, start=first if w else None, rows=prompts * length, max_before=0) for w in windows}
    tab = torch.arange(n * nb, dtype=torch.int32, device=dev).view(n, nb)
    slots = (tab[seq.long(), (pos // bs).long()] * bs + pos % bs).int()
    return StepRows(tokens=torch.zeros(T, dtype=torch.int64, device=dev), pos=pos, slots=slots, tables=tab,
                    states=torch.arange(n, dtype=torch.int32, device=dev), first_pos=first, cu=cu, ctx=ctxs, row_seq=seq,
                    n_portions=prompts, portion_rows=prompts * length, max_portion=length if prompts else 0,
                    max_ctx=ctx + 1, contexts=contexts), n * nb


def kernel_table(s, prompts, length, B, ctx, bs=64):
    """[(phase, kernel, us, ideal us, like kernel, us, ideal us)]"""
    dev = torch.device("cuda")
    hbm, flops, _ = peaks()
    ideal = lambda byts, fl=0.0: max(byts / hbm, fl / flops) * 1e6
    H, G, D, W, width = s["heads"], s["kv"], s["dim"], s["window"], s["width"]
    bf = dict(dtype=torch.bfloat16, device=dev)
    sl = torch.tensor([2.0 ** (-8 * (h + 1) / H) for h in range(H)], device=dev)
    table = []
    # ---- prefill attention
    rows, nb = _rows(prompts, length, 0, 0, bs, dev)
    T = prompts * length
    off = [0, H * D, (H + G) * D, (H + G) * D + s["mh"] * s["mk"], (H + G) * D + 2 * s["mh"] * s["mk"],
           (H + G) * D + 2 * s["mh"] * s["mk"] + s["mh"] * s["mv"]]
    ld = off[5] + s["mh"] * s["mv"]
    projs = [torch.randn(T, ld, **bf) for _ in range(2)]
    cache = torch.zeros(nb, bs, G, D, **bf)
    seen = sum(min(i + 1, W) for i in range(length)) * prompts
    t = graph_us([lambda p=p: wa.window_attention(p, 0, off[1], H, G, D, rows, cache, sl, D ** -0.5, W) for p in projs])
    qkvs = [torch.randn(T, H + 2 * G, D, **bf) for _ in range(2)]
    like = graph_us([lambda p=p: attention.flash_attn_varlen(p[:, :H], p[:, H:H + G], p[:, H + G:], rows.cu, rows.cu, length,
                                                             length, causal=True, window=W) for p in qkvs])
    table.append(("prefill", "window_prefill (+ key append)", t, ideal(T * (2 * H + 3 * G) * D * 2, 4.0 * seen * H * D),
                  "attn_fwd (window)", like, ideal(T * (2 * H + 2 * G) * D * 2, 4.0 * seen * H * D)))
    del qkvs
    # ---- prefill memory
    st = mm.MemoryState.allocate(max(prompts, 1), s["mh"], s["mk"], s["mv"], dev)
    gates, gate_b = torch.randn(T, 2 * s["mh"], device=dev), torch.randn(2 * s["mh"], device=dev)
    o = torch.empty(T, s["mh"], s["mv"], device=dev)
    com = (gate_b, 15.0, s["mk"] ** -0.5, s["mh"], s["mk"], s["mv"])
    t = graph_us([lambda p=p: mm._chunk(p, off[2:5], gates, *com, rows, st, o) for p in projs])
    # the recurrence in chunks of 128: scores and their product with the values inside a chunk, state read and update
    fl = T * s["mh"] * (4.0 * s["mk"] * s["mv"] + 128.0 * (s["mk"] + s["mv"]))
    table.append(("prefill", "matrix_memory_chunk", t,
                  ideal(T * s["mh"] * ((2 * s["mk"] + s["mv"]) * 2 + s["mv"] * 4), fl), None, None, None))
    gain, y = torch.ones(s["mh"] * s["mv"], device=dev), torch.empty(T, s["mh"] * s["mv"], **bf)
    t = graph_us([lambda p=p: mm._output(o, p, off[5], gain, s["mv"], 1e-6, y) for p in projs])
    table.append(("prefill", "memory_output", t, ideal(T * s["mh"] * s["mv"] * 8), None, None, None))
    del projs, o, y
    # ---- residual steps
    for phase, n, cp in (("prefill", T, 2), ("decode", B, 16)):
        xs = [torch.randn(n, width, device=dev) for _ in range(cp)]
        ys = [torch.randn(n, width, **bf) for _ in range(cp)]
        y2 = [torch.randn(n, width, **bf) for _ in range(cp)]
        g = torch.ones(width, device=dev)
        gb = torch.ones(width, **bf)
        like = graph_us([lambda a=a, b=b: fused.rmsnorm(a, gb, 1e-6, b) for a, b in zip(ys, y2)])
        lid = ideal(n * width * 8)
        t = graph_us([lambda x=x, y=y: sandwich.add_sublayer(x, y, g, width, 1e-6, g) for x, y in zip(xs, ys)])
        table.append((phase, "sandwich_norm (one)", t, ideal(n * width * 12), "rmsnorm + residual", like, lid))
        t = graph_us([lambda x=x, y=y, z=z: sandwich.add_sublayer(x, y, g, width, 1e-6, g, y2=z, gain_a=g, gain_b=g)
                      for x, y, z in zip(xs, ys, y2)])
        table.append((phase, "sandwich_norm (pair)", t, ideal(n * width * 14), "rmsnorm + residual", like, lid))
        del xs, ys, y2
    # ---- decode attention
    rows, nb = _rows(0, 0, ctx, B, bs, dev)
    span = min(ctx + 1, W)
    n_c = max(2, math.ceil(3e8 / (B * span * G * D * 2)))
    proj = torch.randn(B, ld, **bf)
    caches = [torch.randn(nb, bs, G, D, **bf) for _ in range(n_c)]
    t = graph_us([lambda c=c: wa.window_attention(proj, 0, off[1], H, G, D, rows, c, sl, D ** -0.5, W) for c in caches])
    vs = [torch.randn(nb, bs, G, D, **bf) for _ in range(n_c)]
    qkv = torch.randn(B, (H + 2 * G) * D, **bf)
    like = graph_us([lambda k=k, v=v: attention.paged_decode_append(qkv, rows.pos, rows.slots, k, v, rows.tables, rows.ctx,
                                                                    ctx + 1, H, G, D, 10000.0, D, window=W)
                     for k, v in zip(caches, vs)])
    table.append(("decode", "shared_kv_decode", t, ideal(B * (span * G + 2 * H) * D * 2, 4.0 * B * span * H * D),
                  "paged_decode (window)", like, ideal(B * (span * 2 * G + 2 * H) * D * 2, 4.0 * B * span * H * D)))
    del caches, vs
    # ---- decode memory
    n_s = max(2, math.ceil(3e8 / (B * s["mh"] * s["mk"] * s["mv"] * 4)))
    sts = [mm.MemoryState.allocate(B, s["mh"], s["mk"], s["mv"], dev) for _ in range(n_s)]
    h, gw = torch.randn(B, width, **bf), torch.randn(2 * s["mh"], width, **bf)
    run = lambda st: mm.matrix_memory(proj, *off[2:6], h, gw, gate_b, 15.0, s["mk"] ** -0.5, s["mh"], s["mk"], s["mv"],
                                      s["mv"], rows, st, gain, 1e-6)
    t = graph_us([lambda st=st: run(st) for st in sts])
    table.append(("decode", "matrix_memory step", t, ideal(2 * B * s["mh"] * s["mk"] * s["mv"] * 4), None, None,
                  None))
    return table


def _families():
    from . import serve_bench_kedesun as sk, serve_bench_lobutar as sl, serve_bench_rezulorn as sr
    active = lambda eng, s, n: n - 2 * VOCAB * s["width"]
    return {"nafitar": dict(like="dense", sizes=SIZES, active=active, table=kernel_table,
                            decode_bytes=lambda kind, s, eng, B, ctx: decode_bytes(kind, s, eng, B, ctx)),
            "kedesun": dict(like="latent", sizes=sk.SIZES, active=sk.active_weights, table=sk.kernel_table,
                            decode_bytes=sk.decode_bytes),
            "lobutar": dict(like="grouped", sizes=sl.SIZES, active=sl.active_weights, table=sl.kernel_table,
                            decode_bytes=sl.decode_bytes),
            "rezulorn": dict(like=("nafitar", "mixed"), sizes=sr.SIZES, active=sr.active_weights, table=sr.kernel_table,
                             decode_bytes=sr.decode_bytes)}


def run(sizes=None, iters=10, design="nafitar"):
    hbm, flops, which = peaks()
    fam = _families()[design]
    out = {"design": design, "peaks": which, "gpu": torch.cuda.get_device_name(0), "dtype": "bf16", "data": "synthetic",
           "sizes": {}}
    prompts, length, ctx = 4, 4096, 4096
    for name in sizes or fam["sizes"]:
        s = fam["sizes"][name]
        rec = {"layer": s, "prefill": {}, "decode": {}}
        for kind in (design, *((fam["like"],) if isinstance(fam["like"], str) else fam["like"])):
            eng = build(kind, s, ctx + 256, 64)
            n_params = sum(t.numel() for t in eng.w.tensors())
            ms = prefill_step(eng, prompts, length, max(3, iters // 2))
            T = prompts * length
            rec["prefill"][kind] = {"ms": round(ms, 3), "tokens_per_s": round(T / ms * 1e3),
                                    "gemm_roofline_fraction": round(2.0 * T * fam["active"](eng, s, n_params) / flops
                                                                    / (ms * 1e-3), 3)}
            for B in (8, 64):
                ms = decode_step(eng, B, ctx, iters * 3)
                rec["decode"][f"{kind}_b{B}"] = {"ms": round(ms, 4), "tokens_per_s": round(B / ms * 1e3),
                                                 "hbm_roofline_fraction": round(fam["decode_bytes"](kind, s, eng, B, ctx)
                                                                                / hbm / (ms * 1e-3), 3)}
            del eng
            torch.cuda.empty_cache()
        rec["kernels"] = []
        for B in (8, 64):
            for phase, k, t, i, lk, lt, li in fam["table"](s, prompts, length, B, ctx):
                if phase == "prefill" and B != 8:
                    continue
                r = {"phase": phase if phase == "prefill" else f"{phase} b{B}", "kernel": k, "us": round(t, 2),
                     "ideal_us": round(i, 2), "distance": round(t / i, 2)}
                if lk:
                    r.update(like=lk, like_us=round(lt, 2), like_ideal_us=round(li, 2), like_distance=round(lt / li, 2),
                             ratio=round((t / i) / (lt / li), 2))
                rec["kernels"].append(r)
            torch.cuda.empty_cache()
        out["sizes"][name] = rec
    _lib.check_device_errors()
    return out

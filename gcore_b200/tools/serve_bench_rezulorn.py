"""Rezulorn's part of the serving benchmark (``serve_bench.py``): layer sizes, the decoders it is compared with (Nafitar, which
also runs attention and a recurrent memory side by side, and a dense grouped-query decoder), and its kernels beside the like
kernels of those."""
from __future__ import annotations

import math

import torch

from ..models.config import ModelConfig
from ..ops import attention, fused, head_prep as hp, moe, sandwich
from ..ops import conv_norm as cn
from ..ops import matrix_memory as mm
from ..ops import scored_attention as sa

# width, heads, kv heads and head size of both attentions, window and kept positions of one, heads and sizes of the retention
# beside the other (rh, rk, rv) and of the lightning layers (lh, lk, lv), feed-forward (two matrices; nff: three of the compared
# models, equal weight), layers (parallel, lightning, attention in turn); mh, mk, mv: Nafitar's memory
SIZES = {
    "2k": dict(width=2048, heads=16, kv=4, dim=128, window=1024, keep=16, rh=8, rk=128, rv=256, lh=16, lk=128, lv=128, ff=8448,
               nff=5632, layers=12, taps=4, mh=8, mk=128, mv=256),
    "4k": dict(width=4096, heads=32, kv=8, dim=128, window=2048, keep=64, rh=16, rk=128, rv=256, lh=32, lk=128, lv=128, ff=16512,
               nff=11008, layers=9, taps=4, mh=16, mk=128, mv=256),
    "3k-small-heads": dict(width=3072, heads=48, kv=8, dim=64, window=1024, keep=4, rh=12, rk=64, rv=128, lh=24, lk=64, lv=128,
                           ff=12288, nff=8192, layers=9, taps=3, mh=12, mk=64, mv=128),
}


def _decay(n):
    return [1 - 2.0 ** (-4 - 6 * h / max(n - 1, 1)) for h in range(n)]


def conf(s):
    from .serve_bench import VOCAB
    heads, rot = dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["dim"], scale=s["dim"] ** -0.5), dict(base=1e4)
    kinds = [dict(type="parallel", mixer=dict(
        left=dict(heads, rot=dict(rot, dims=s["dim"])), left_scale=0.5, right_scale=0.5,
        right=dict(heads=s["rh"], dim=s["rk"], vdim=s["rv"], decay=_decay(s["rh"]), rot=dict(rot, dims=s["rk"])))),
        dict(type="lightning", mixer=dict(heads=s["lh"], dim=s["lk"], vdim=s["lv"], decay=_decay(s["lh"]))),
        dict(type="attention", mixer=dict(heads, mask=dict(size=s["window"], keep_first=s["keep"])))]
    return dict(architecture="Rezulorn", canon=dict(taps=s["taps"]), logit_scale=1.0, residual_mult=0.5, norm=dict(eps=1e-6),
                layers=[dict(kinds[i % 3], mlp=dict(kind="dense", ff=s["ff"])) for i in range(s["layers"])], vocab=VOCAB,
                width=s["width"])


def like_sizes(s):
    return dict(s, ff=s["nff"])


def dense_config(s):
    """Attention in every layer, a third of them in a window."""
    from .serve_bench import VOCAB
    return ModelConfig(arch="llama", num_layers=s["layers"], hidden_size=s["width"], num_attention_heads=s["heads"],
                       num_kv_heads=s["kv"], head_dim=s["dim"], ffn_hidden_size=s["nff"], vocab_size=VOCAB, qkv_bias=True,
                       sliding_window=s["window"], sliding_window_pattern=[0, 0, 1])


def active_weights(eng, s, n):
    from .serve_bench import VOCAB
    return n - 2 * VOCAB * s["width"]


def decode_bytes(kind, s, eng, B, ctx):
    """HBM bytes one decode step has to move: weights once, the cached rows that are seen, recurrent state in and out."""
    from .serve_bench import decode_bytes as base, model_bytes
    if kind == "nafitar":
        return base(kind, s, eng, B, ctx)
    L, row = s["layers"] // 3, 2 * s["kv"] * s["dim"] * 2
    span = min(ctx + 1, s["window"] + s["keep"])
    if kind != "rezulorn":
        return model_bytes(eng) + B * row * L * (2 * (ctx + 1) + min(ctx + 1, s["window"]))
    state = s["rh"] * s["rk"] * s["rv"] + s["lh"] * s["lk"] * s["lv"]
    ring = 6 * s["taps"] * s["width"]                 # taps - 1 rows read and one written, two sublayers, three layers
    return model_bytes(eng) + B * L * (row * (ctx + 1 + span) + 4 * (2 * state + ring))


def kernel_table(s, prompts, length, B, ctx, bs=64):
    """[(phase, kernel, us, ideal us, like kernel, us, ideal us)]"""
    from ..models.layer_plan import RetentionSpec, RotarySpec, ScoredAttentionSpec
    from ..models.plan_modules import RetentionMixer, ScoredAttentionMixer
    from .serve_bench import _rows, graph_us, peaks
    dev = torch.device("cuda")
    hbm, flops, _ = peaks()
    ideal = lambda byts, fl=0.0: max(byts / hbm, fl / flops) * 1e6
    bf, f32 = dict(dtype=torch.bfloat16, device=dev), dict(dtype=torch.float32, device=dev)
    H, G, D, W, K, width = s["heads"], s["kv"], s["dim"], s["window"], s["keep"], s["width"]
    mod = dict(width=width, eps=1e-6, dtype=torch.bfloat16, device=dev, out_scale=0.5)
    sig = ScoredAttentionMixer(ScoredAttentionSpec(H, G, D, D, D ** -0.5, weights="sigmoid", rot=RotarySpec(D, 1e4, halves=True),
                                                   unit=True, head_bias=True), **mod)
    dis = ScoredAttentionMixer(ScoredAttentionSpec(H, G, D, D, D ** -0.5, distance=True, window=W, keep=K), **mod)
    sig.head_bias.fill_(-4.0)
    dis.r1.fill_(0.5)
    dis.r2.fill_(0.5)
    ret = RetentionMixer(RetentionSpec(s["rh"], s["rk"], s["rv"], tuple(_decay(s["rh"])), rot=RotarySpec(s["rk"], 1e4)), **mod)
    lig = RetentionMixer(RetentionSpec(s["lh"], s["lk"], s["lv"], tuple(_decay(s["lh"])), scale=1.0, act="silu", norm="joint",
                                       gate="sigmoid"), **mod)
    lig.gain.fill_(1.0)
    table = []
    # ---- prompts: attention
    rows, nb = _rows(prompts, length, 0, 0, bs, dev)
    T = prompts * length
    qkvs = [torch.randn(T, (H + 2 * G) * D, **bf) for _ in range(2)]
    out = torch.empty(T, H * D, **bf)
    cache = torch.zeros(nb, bs, 2 * G * D, **bf)
    kc, vc = (torch.zeros(nb, bs, G, D, **bf) for _ in range(2))
    ly = sig.layout
    t = graph_us([lambda p=p: sa._prepare(p, ly, sig.turns, rows, 0, T, cache) for p in qkvs])
    like = graph_us([lambda p=p: attention.kv_append_rope(p, rows.pos, rows.slots, kc, vc, H, G, D, 10000.0, D) for p in qkvs])
    i = ideal(T * (2 * H + 4 * G) * D * 2)
    table.append(("prefill", "head_prep (rotate, norm, append)", t, i, "kv_append_rope", like, i))
    prepare, sa._prepare = sa._prepare, lambda *a: None      # the attention kernels alone
    views = [p.view(T, H + 2 * G, D) for p in qkvs]
    byts = T * (2 * H + 2 * G) * D * 2
    try:
        for mix, name, window in ((sig, "scored_prefill (sigmoid)", 0), (dis, "scored_prefill (distance, window)", W)):
            kw = (mix.turns, (mix.r1, mix.r2) if mix.r1 is not None else None, mix.head_bias)
            t = graph_us([lambda p=p: sa._portions(p, mix.layout, *kw, rows, cache, out, 0.5) for p in qkvs])
            like = graph_us([lambda p=p: attention.flash_attn_varlen(p[:, :H], p[:, H:H + G], p[:, H + G:], rows.cu, rows.cu,
                                                                     length, length, causal=True, window=window) for p in views])
            full = prompts * length * (length + 1) / 2
            far = prompts * sum(min(i + 1, window) for i in range(length)) if window else full
            kept = prompts * sum(min(max(i + 1 - window, 0), K) for i in range(length)) if window else 0
            table.append(("prefill", name, t, ideal(byts, 4.0 * (far + kept) * H * D),
                          "attn_fwd (window)" if window else "attn_fwd", like, ideal(byts, 4.0 * far * H * D)))
    finally:
        sa._prepare = prepare
    del qkvs, views, out, kc, vc
    # ---- prompts: memories
    mh, mk, mv = s["mh"], s["mk"], s["mv"]
    proj = [torch.randn(T, 2 * mh * (mk + mv), **bf) for _ in range(2)]
    gates, gate_b, o = torch.randn(T, 2 * mh, **f32), torch.randn(2 * mh, **f32), torch.empty(T, mh, mv, **f32)
    st = mm.MemoryState.allocate(prompts, mh, mk, mv, dev)
    offs = (0, mh * mk, 2 * mh * mk)
    mlike = graph_us([lambda p=p: mm._chunk(p, offs, gates, gate_b, 15.0, mk ** -0.5, mh, mk, mv, rows, st, o) for p in proj])
    fl = lambda h, k, v: T * h * (4.0 * k * v + 128.0 * (k + v))
    mid = ideal(T * mh * ((2 * mk + mv) * 2 + mv * 4), fl(mh, mk, mv))
    gain, y = torch.ones(mh * mv, **f32), torch.empty(T, mh * mv, **bf)
    olike = graph_us([lambda p=p: mm._output(o, p, offs[2] + mh * mv, gain, mv, 1e-6, y) for p in proj])
    oid = ideal(T * mh * mv * 8)
    del proj, gates, o, y, st
    for mix, name in ((ret, "retention"), (lig, "lightning")):
        sp = mix.spec
        h, k, v = sp.heads, mix.dim, mix.vdim
        proj = [torch.randn(T, mix.columns, **bf) for _ in range(2)]
        o, y, st = torch.empty(T, h, v, **f32), torch.empty(T, h * v, **bf), mix.new_state(prompts, dev)
        if mix.turns is not None:
            t = graph_us([lambda p=p: hp.head_prep(p, rows, 0, T, mix.at[0], h, mix.at[1], h, k, turns=mix.turns) for p in proj])
            table.append(("prefill", f"head_prep ({name}: rotate)", t, ideal(T * h * k * 8), None, None, None))
        else:
            n = mix.at[3]
            t = graph_us([lambda p=p: hp.silu_columns(p, 0, n) for p in proj])
            gu = [torch.randn(T, 2 * n, **bf) for _ in range(2)]
            like = graph_us([lambda p=p: fused.swiglu(p) for p in gu])
            table.append(("prefill", f"silu_columns ({name})", t, ideal(T * n * 4), "swiglu", like, ideal(T * n * 6)))
            del gu
        t = graph_us([lambda p=p: mm._chunk(p, tuple(mix.at[:3]), None, None, 0.0, 1.0, h, k, v, rows, st, o, mix.decay)
                      for p in proj])
        table.append(("prefill", f"memory chunk ({name})", t, ideal(T * h * ((2 * k + v) * 2 + v * 4), fl(h, k, v)),
                      "matrix_memory_chunk", mlike, mid))
        t = graph_us([lambda p=p: mm._output(o, p, mix.at[3], mix.gain, sp.vdim, 1e-6, y, mix.gain is not None, 0.5)
                      for p in proj])
        table.append(("prefill", f"memory output ({name})", t, ideal(T * h * v * 8), "memory_output", olike, oid))
        del proj, o, y, st
    # ---- residual steps, activation
    spec, taps = cn.NormSpec(width, 1e-6), torch.randn(cn.stored_taps(s["taps"]), width, **f32)
    gain, gb = torch.ones(width, **f32), torch.ones(width, **bf)
    single, _ = _rows(0, 0, ctx, B, bs, dev)
    for phase, n, rw, cp in (("prefill", T, rows, 2), ("decode", B, single, 16)):
        xs, ys = [torch.randn(n, width, **f32) for _ in range(cp)], [torch.randn(n, width, **bf) for _ in range(cp)]
        rings = [torch.zeros(rw.states.numel(), taps.shape[0] - 1, width, **f32) for _ in range(cp)]
        t = graph_us([lambda x=x, y=y, r=r: cn.conv_add_sublayer(x, y, 0.5, spec, gain, rw, taps, r)
                      for x, y, r in zip(xs, ys, rings)])
        like = graph_us([lambda x=x, y=y: sandwich.add_sublayer(x, y, gain, width, 1e-6, gain) for x, y in zip(xs, ys)])
        state = rw.states.numel() * (taps.shape[0] - 1 + min(n // rw.states.numel(), taps.shape[0] - 1)) * width * 4
        table.append((phase, f"conv_norm ({s['taps']} taps)", t, ideal(n * width * 12 + state), "sandwich_norm (one)", like,
                      ideal(n * width * 12)))
        del xs, ys, rings
        us, gu = [torch.randn(n, s["ff"], **bf) for _ in range(2)], [torch.randn(n, 2 * s["nff"], **bf) for _ in range(2)]
        dst = torch.empty_like(us[0])
        t = graph_us([lambda u=u: moe.activate(moe.RELU2, u, s["ff"], 0, dst) for u in us])
        like = graph_us([lambda g=g: fused.swiglu(g) for g in gu])
        table.append((phase, "squared relu", t, ideal(n * s["ff"] * 4), "swiglu", like, ideal(n * s["nff"] * 6)))
        del us, gu, dst
    # ---- decode: attention
    rows, nb = _rows(0, 0, ctx, B, bs, dev)
    proj, out = torch.randn(B, (H + 2 * G) * D, **bf), torch.empty(B, H * D, **bf)
    for mix, name, window in ((sig, "scored_decode (sigmoid)", 0), (dis, "scored_decode (distance, window)", W)):
        span = min(ctx + 1, window + K) if window else ctx + 1
        n_c = max(2, math.ceil(3e8 / (B * span * 2 * G * D * 2)))
        caches = [torch.randn(nb, bs, 2 * G * D, **bf) for _ in range(n_c)]
        kw = (mix.turns, (mix.r1, mix.r2) if mix.r1 is not None else None, mix.head_bias)
        t = graph_us([lambda c=c: sa._decode(proj, mix.layout, *kw, rows, c, out, 0.5) for c in caches])
        del caches
        ks, vs = ([torch.randn(nb, bs, G, D, **bf) for _ in range(n_c)] for _ in range(2))
        like = graph_us([lambda k=k, v=v: attention.paged_decode_append(proj, rows.pos, rows.slots, k, v, rows.tables, rows.ctx,
                                                                        ctx + 1, H, G, D, 10000.0, D, window=window)
                         for k, v in zip(ks, vs)])
        del ks, vs
        i = lambda n: ideal(B * (n * 2 * G + 2 * H) * D * 2, 4.0 * B * n * H * D)
        table.append(("decode", name, t, i(span), "paged_decode (window)" if window else "paged_decode", like,
                      i(min(ctx + 1, window) if window else ctx + 1)))
    # ---- decode: memories
    n_s = max(2, math.ceil(3e8 / (B * mh * mk * mv * 4)))
    sts = [mm.MemoryState.allocate(B, mh, mk, mv, dev) for _ in range(n_s)]
    proj, h = torch.randn(B, 2 * mh * (mk + mv), **bf), torch.randn(B, width, **bf)
    gw, gain = torch.randn(2 * mh, width, **bf), torch.ones(mh * mv, **f32)
    mlike = graph_us([lambda st=st: mm.matrix_memory(proj, *offs, offs[2] + mh * mv, h, gw, gate_b, 15.0, mk ** -0.5, mh, mk, mv,
                                                     mv, rows, st, gain, 1e-6) for st in sts])
    mid = ideal(2 * B * mh * mk * mv * 4)
    del sts
    for mix, name in ((ret, "retention"), (lig, "lightning")):
        size = mix.spec.heads * mix.dim * mix.vdim
        sts = [mix.new_state(B, dev) for _ in range(max(2, math.ceil(3e8 / (B * size * 4))))]
        proj, out = torch.randn(B, mix.columns, **bf), torch.empty(B, mix.out_columns, **bf)
        t = graph_us([lambda st=st: mix(proj, rows, None, st, out) for st in sts])
        table.append(("decode", f"memory step ({name})", t, ideal(2 * B * size * 4), "matrix_memory step", mlike, mid))
        del sts
    return table

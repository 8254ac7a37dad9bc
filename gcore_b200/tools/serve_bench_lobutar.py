"""Lobutar's part of the serving benchmark (``serve_bench.py``): layer sizes, the latent-attention decoder with experts it is
compared with, and its kernels beside the like kernels of the framework's other models."""
from __future__ import annotations

import math

import torch

from ..models.config import ModelConfig
from ..ops import attention, fused, moe
from ..ops import diff_attention as da
from ..ops import latent_attention as la
from ..ops import streams as hc
from ..ops.router import route

# width, heads and kv heads of the differential attention, its map and value sizes, heads and sizes of the latent attention
# (unrotated, rotated, value, latent) and its window, dense and expert feed-forwards, streams, layers (every fourth is latent
# attention, the first has the dense feed-forward)
SIZES = {
    "2k": dict(width=2048, heads=16, kv=4, dim=64, vdim=128, lh=16, ldim=128, lrot=64, lv=128, rank=512, window=1024, ff=5632,
               experts=32, top=4, eff=1024, groups=8, keep=4, streams=4, layers=8),
    "4k": dict(width=4096, heads=32, kv=8, dim=64, vdim=128, lh=32, ldim=128, lrot=64, lv=128, rank=512, window=2048, ff=11008,
               experts=64, top=4, eff=1536, groups=8, keep=4, streams=2, layers=8),
    "3k-wide-maps": dict(width=3072, heads=12, kv=6, dim=128, vdim=256, lh=24, ldim=64, lrot=32, lv=64, rank=128, window=512,
                         ff=8192, experts=32, top=2, eff=2048, groups=4, keep=2, streams=3, layers=8),
}


def conf(s):
    from .serve_bench import VOCAB
    dense = dict(kind="dense", ff=s["ff"])
    expert = dict(kind="moe", expert=dict(ff=s["eff"]), shared=dict(ff=s["eff"]),
                  router=dict(experts=s["experts"], top=s["top"], scale=1.5, groups=dict(count=s["groups"], keep=s["keep"])))
    layers = []
    for i in range(s["layers"]):
        if i % 4 == 3:
            m = dict(type="latent_attention", mixer=dict(
                heads=s["lh"], dim=s["ldim"], rot_dim=s["lrot"], vdim=s["lv"], kv_rank=s["rank"], mask=dict(size=s["window"]),
                scale=(s["ldim"] + s["lrot"]) ** -0.5, rot=dict(dims=s["lrot"], base=10000.0)))
        else:
            m = dict(type="attention", mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["vdim"], diff=0.4,
                                                  scale=s["dim"] ** -0.5, rot=dict(dims=s["dim"] // 2, base=10000.0)))
        layers.append(dict(m, mlp=expert if i else dense))
    return dict(architecture="Lobutar", layers=layers, norm=dict(eps=1e-6), streams=s["streams"], vocab=VOCAB, width=s["width"])


def latent_config(s):
    """Latent attention in every layer, the same feed-forwards."""
    from .serve_bench import VOCAB
    return ModelConfig(arch="deepseek_v3", num_layers=s["layers"], hidden_size=s["width"], num_attention_heads=s["lh"],
                       num_kv_heads=s["lh"], head_dim=192, ffn_hidden_size=s["ff"], vocab_size=VOCAB, use_mla=True,
                       q_lora_rank=0, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                       num_experts=s["experts"], moe_top_k=s["top"], moe_ffn_hidden_size=s["eff"],
                       moe_shared_expert_ffn=s["eff"], first_k_dense=1, moe_router_type="sigmoid_group",
                       moe_n_group=s["groups"], moe_topk_group=s["keep"], moe_norm_topk_prob=True, moe_router_bias=True)


def _idle_experts(s, used):
    """Weights of the routed experts beyond ``used`` per expert layer."""
    return (s["layers"] - 1) * (s["experts"] - used) * 3 * s["eff"] * s["width"]


def active_weights(eng, s, n):
    """Weights a token is multiplied with, without the vocabulary matrices."""
    cfg = eng.cfg
    if eng.plan is None:
        return cfg.active_parameters() - 2 * cfg.vocab_size * cfg.hidden_size
    return cfg.num_parameters(include_embedding=False) - _idle_experts(s, s["top"])


def decode_bytes(kind, s, eng, B, ctx):
    """HBM bytes one decode step has to move: weights once (of the experts, those that B tokens choose at random), and the
    cached rows that are seen."""
    cfg = eng.cfg
    hit = s["experts"] * (1 - (1 - s["top"] / s["experts"]) ** B)
    w = cfg.num_parameters(include_embedding=False) + cfg.vocab_size * cfg.hidden_size - _idle_experts(s, hit)
    if kind != "lobutar":
        return 2 * w + s["layers"] * B * (ctx + 1) * 576 * 2
    n_lat = s["layers"] // 4
    cache = n_lat * B * min(ctx + 1, s["window"]) * (s["rank"] + s["lrot"])
    cache += (s["layers"] - n_lat) * B * (ctx + 1) * s["kv"] * (2 * s["dim"] + s["vdim"])
    return 2 * (w + cache)


def _mixers(s, dev):
    from ..models.layer_plan import DifferentialAttentionSpec, LatentAttentionSpec, RotarySpec
    from ..models.plan_modules import DifferentialAttentionMixer, LatentAttentionMixer
    d = DifferentialAttentionMixer(DifferentialAttentionSpec(s["heads"], s["kv"], s["dim"], s["vdim"], s["dim"] ** -0.5, 0.4,
                                                             RotarySpec(s["dim"] // 2, 10000.0)), s["width"], 1e-6,
                                   torch.bfloat16, dev)
    d.lam.fill_(0.5)
    m = LatentAttentionMixer(LatentAttentionSpec(s["lh"], s["ldim"], s["lrot"], s["lv"], s["rank"],
                                                 (s["ldim"] + s["lrot"]) ** -0.5, RotarySpec(s["lrot"], 10000.0), s["window"],
                                                 True, "element"), s["width"], 1e-6, torch.bfloat16, dev)
    m.up_kv.normal_(0, s["rank"] ** -0.5)
    m.gain.fill_(1.0)
    return d, m


def kernel_table(s, prompts, length, B, ctx, bs=64):
    """[(phase, kernel, us, ideal us, like kernel, us, ideal us)]"""
    from .serve_bench import _rows, graph_us, peaks
    dev = torch.device("cuda")
    hbm, flops, _ = peaks()
    ideal = lambda byts, fl=0.0: max(byts / hbm, fl / flops) * 1e6
    bf, f32 = dict(dtype=torch.bfloat16, device=dev), dict(dtype=torch.float32, device=dev)
    H, G, dim, vdim, W, width = s["heads"], s["kv"], s["dim"], s["vdim"], s["window"], s["width"]
    D = 128                                         # head size of the compared grouped-query attention
    dif, lat = _mixers(s, dev)
    dl, ll = dif.layout, lat.layout
    table = []
    # ---- prompt: differential attention
    rows, nb = _rows(prompts, length, 0, 0, bs, dev, (W,))
    T = prompts * length
    projs = [torch.randn(T, dif.columns, **bf) for _ in range(2)]
    cache = torch.zeros(nb, bs, dl.row, **bf)
    out = torch.empty(T, dif.out_columns, **bf)
    t = graph_us([lambda p=p: da._append(p, dl, dif.turns, rows, 0, T, cache) for p in projs])
    qkvs = [torch.randn(T, (H + 2 * G) * D, **bf) for _ in range(2)]
    kc, vc = (torch.zeros(nb, bs, G, D, **bf) for _ in range(2))
    like = graph_us([lambda p=p: attention.kv_append_rope(p, rows.pos, rows.slots, kc, vc, H, G, D, 10000.0, dim // 2)
                     for p in qkvs])
    table.append(("prefill", "rotate_append", t, ideal(T * (2 * H * dl.rot * 2 + 2 * dl.row) * 2), "kv_append_rope", like,
                  ideal(T * (H * (dim // 2) * 2 + 4 * G * D) * 2)))
    append, da._append = da._append, lambda *a: None      # the attention kernel alone
    try:
        t = graph_us([lambda p=p: da._portions(p, dl, dif.turns, dif.lam, rows, cache, out) for p in projs])
    finally:
        da._append = append
    pairs = prompts * length * (length + 1) / 2
    qkv = [p.view(T, H + 2 * G, D) for p in qkvs]
    like = graph_us([lambda p=p: attention.flash_attn_varlen(p[:, :H], p[:, H:H + G], p[:, H + G:], rows.cu, rows.cu, length,
                                                             length, causal=True) for p in qkv])
    table.append(("prefill", "diff_prefill", t, ideal(T * (2 * H * dim + dl.row + H * vdim) * 2, 4.0 * pairs * H * (dim + vdim)),
                  "attn_fwd 128/128", like, ideal(T * (2 * H + 2 * G) * D * 2, 4.0 * pairs * H * D)))
    del projs, qkvs, qkv, kc, vc, out
    # ---- prompt: latent attention
    lh, ldim, lrot, lv, rank = s["lh"], s["ldim"], s["lrot"], s["lv"], s["rank"]
    projs = [torch.randn(T, lat.columns, **bf) for _ in range(2)]
    cache = torch.zeros(nb, bs, ll.row, **bf)
    context, kv = torch.randn(T, ll.row, **bf), torch.randn(T, lh * (ldim + lv), **bf)
    out = torch.empty(T, lat.out_columns, **bf)
    la_linear = la.linear_forward
    la.linear_forward = lambda *a: kv            # the attention kernel alone
    try:
        t = graph_us([lambda p=p: la._portions(p, ll, lat.up_kv, rows, cache, context, out, lat.sinks) for p in projs])
    finally:
        la.linear_forward = la_linear
    seen = prompts * sum(min(i + 1, W) for i in range(length))
    fl = 2.0 * seen * lh * (ldim + lrot + lv)
    qk, v = [torch.randn(T, 2 * lh, 192, **bf) for _ in range(2)], torch.randn(T, lh, 128, **bf)
    like = graph_us([lambda a=a: attention.flash_attn_varlen(a[:, :lh], a[:, lh:], v, rows.cu, rows.cu, length, length,
                                                             causal=True, window=W) for a in qk])
    table.append(("prefill", "latent attention (window, sink, gate)", t, ideal(T * lh * (2 * ldim + lrot + 3 * lv) * 2, fl),
                  "attn_fwd 192/128 (window)", like, ideal(T * lh * 640 * 2, 2.0 * seen * lh * 320)))
    del projs, qk, v, kv, context, out
    # ---- streams, experts: prompt and decode
    S, E, K = s["streams"], s["experts"], s["top"]
    for phase, n, cp in (("prefill", T, 2), ("decode", B, 8)):
        xs = [torch.randn(n, S, width, **f32) for _ in range(cp)]
        ys = [torch.randn(n, width, **bf) for _ in range(cp)]
        mix, one, gain, gb = torch.eye(S, **f32), torch.ones(S, **f32) / S, torch.ones(width, **f32), torch.ones(width, **bf)
        like = graph_us([lambda a=a, b=b: fused.rmsnorm(a, gb, 1e-6, b) for a, b in zip(ys, ys[1:] + ys[:1])])
        lid = ideal(n * width * 8)
        t = graph_us([lambda x=x, y=y: hc.connect(x, y, mix, one, width, 1e-6, one, gain) for x, y in zip(xs, ys)])
        table.append((phase, f"stream_mix ({S})", t, ideal(n * width * (8 * S + 4)), "rmsnorm + residual", like, lid))
        er = torch.randn(n * K, width, **bf)
        dest, w = torch.randperm(n * K, device=dev).int().view(n, K), torch.rand(n, K, **f32)
        t = graph_us([lambda x=x, y=y: hc.connect(x, y, mix, one, width, 1e-6, one, gain, (er, dest, w))
                      for x, y in zip(xs, ys)])
        table.append((phase, f"stream_mix ({S}, {K} experts)", t, ideal(n * width * (8 * S + 4 + 2 * K)), "rmsnorm + residual",
                      like, lid))
        del xs, er
        corr, counts = torch.zeros(E, **f32), torch.zeros(E, dtype=torch.int32, device=dev)
        router = torch.randn(E, width, **bf)
        rw = router.float()
        how = dict(sigmoid=True, norm=False, scale=1.5, groups=s["groups"], keep=s["keep"])
        t = graph_us([lambda y=y: moe.route_tokens(y, router, E, K, corr, counts, **how) for y in ys])
        like = graph_us([lambda y=y: route(torch.nn.functional.linear(y.float(), rw), corr, None, K, s["groups"], s["keep"],
                                           True, True, 1.5) for y in ys])
        i = ideal((n + E) * width * 2)
        table.append((phase, "logits + grouped choice", t, i, "logits + route", like, i))
        del ys
        torch.cuda.empty_cache()
    # ---- decode: differential attention
    rows, nb = _rows(0, 0, ctx, B, bs, dev)
    n_c = max(2, math.ceil(3e8 / (B * (ctx + 1) * dl.row * 2)))
    proj, out = torch.randn(B, dif.columns, **bf), torch.empty(B, dif.out_columns, **bf)
    caches = [torch.randn(nb, bs, dl.row, **bf) for _ in range(n_c)]
    t = graph_us([lambda c=c: da._decode(proj, dl, dif.turns, dif.lam, rows, c, out) for c in caches])
    del caches
    n_c = max(2, math.ceil(3e8 / (B * (ctx + 1) * G * D * 4)))
    kcs, vcs = ([torch.randn(nb, bs, G, D, **bf) for _ in range(n_c)] for _ in range(2))
    qkv = torch.randn(B, (H + 2 * G) * D, **bf)
    like = graph_us([lambda k=k, v=v: attention.paged_decode_append(qkv, rows.pos, rows.slots, k, v, rows.tables, rows.ctx,
                                                                    ctx + 1, H, G, D, 10000.0, D) for k, v in zip(kcs, vcs)])
    table.append(("decode", "diff_decode", t, ideal(B * ((ctx + 1) * dl.row + H * (2 * dim + vdim)) * 2,
                                                    4.0 * B * (ctx + 1) * H * (dim + vdim)),
                  "paged_decode (with append)", like, ideal(B * ((ctx + 1) * G + H) * 2 * D * 2,
                                                            4.0 * B * (ctx + 1) * H * D)))
    del kcs, vcs
    # ---- decode: latent attention in a window, and the gate behind it
    span = min(W, ctx + 1)
    n_c = max(2, math.ceil(3e8 / (B * span * ll.row * 2)))
    proj, out = torch.randn(B, lat.columns, **bf), torch.empty(B, lat.out_columns, **bf)
    caches = [torch.randn(nb, bs, ll.row, **bf) for _ in range(n_c)]
    bmm, la._bmm = la._bmm, lambda a, b, out: out      # the attention and gate kernels alone
    try:
        t = graph_us([lambda c=c: la._absorbed(proj, ll, lat.up_kv, rows, 0, B, c, out, lat.sinks) for c in caches])
    finally:
        la._bmm = bmm
    short, _ = _rows(0, 0, span - 1, B, bs, dev)
    q_lat, q_rope = torch.randn(lh, B, ll.row_rank, **bf), torch.randn(B, lh, ll.row_rot, **bf)
    o_lat = torch.empty_like(q_lat)
    like = graph_us([lambda c=c: attention.mla_paged_decode(q_lat.transpose(0, 1), q_rope, c, short.tables, short.ctx, span,
                                                            lat.spec.scale, out=o_lat.transpose(0, 1)) for c in caches])
    i = ideal(B * span * ll.row * 2 + B * lh * (2 * ll.row_rank + lrot) * 2, 2.0 * B * span * lh * (2 * ll.row_rank + ll.row_rot))
    table.append(("decode", "mla_paged_decode (window, sink) + gate", t, i, "mla_paged_decode (no window)", like, i))
    return table

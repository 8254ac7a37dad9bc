"""Kedesun's part of the serving benchmark (``serve_bench.py``): layer sizes, the latent-attention decoder with experts it is
compared with, and its kernels beside the like kernels of the framework's other models."""
from __future__ import annotations

import math

import torch

from ..models.config import ModelConfig
from ..models.moe import build_dispatch_plan, padded_rows_bound
from ..ops import attention, depth, fused, moe
from ..ops import latent_attention as la
from ..ops import matrix_memory as mm
from ..ops.gemm import grouped_gemm
from ..ops.router import route

# width, attention heads and head sizes (unrotated, rotated, value), latent size, retention heads and sizes, dense and
# expert feed-forwards, layers (every fourth layer is latent attention; feed-forwards alternate between dense and experts)
SIZES = {
    "2k": dict(width=2048, heads=16, dim=128, rot=64, vdim=128, rank=512, rh=8, rk=128, rv=256, ff=5632, experts=32, top=4,
               eff=1024, layers=12),
    "4k": dict(width=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, rh=16, rk=128, rv=256, ff=11008, experts=64, top=4,
               eff=1536, layers=8),
    "3k-wide-keys": dict(width=3072, heads=24, dim=128, rot=64, vdim=128, rank=256, rh=6, rk=256, rv=512, ff=8192, experts=32,
                         top=2, eff=2048, layers=8),
}


def conf(s):
    from .serve_bench import VOCAB
    dense = dict(kind="dense", ff=s["ff"])
    expert = dict(kind="moe", expert=dict(ff=s["eff"]), shared=dict(ff=s["eff"]),
                  router=dict(experts=s["experts"], top=s["top"]))
    layers = []
    for i in range(s["layers"]):
        if i % 4 == 3:
            m = dict(type="latent_attention", mixer=dict(
                heads=s["heads"], dim=s["dim"], rot_dim=s["rot"], vdim=s["vdim"], kv_rank=s["rank"],
                scale=(s["dim"] + s["rot"]) ** -0.5,
                rot=dict(dims=s["rot"], base=10000.0, scaling=dict(factor=4.0, original=1024, fast=32.0, slow=1.0))))
        else:
            m = dict(type="retention", mixer=dict(heads=s["rh"], dim=s["rk"], vdim=s["rv"],
                                                  decay=[1 - 2.0 ** (-5 - h) for h in range(s["rh"])]))
        layers.append(dict(m, mlp=expert if i % 2 else dense))
    return dict(architecture="Kedesun", layers=layers, norm=dict(eps=1e-6), vocab=VOCAB, width=s["width"])


def latent_config(s):
    """Latent attention in every layer, the same feed-forwards; gated experts of two thirds the width hold as much."""
    from .serve_bench import VOCAB
    ff = s["eff"] * 2 // 3 // 64 * 64
    return ModelConfig(arch="deepseek_v3", num_layers=s["layers"], hidden_size=s["width"], num_attention_heads=s["heads"],
                       num_kv_heads=s["heads"], head_dim=s["dim"] + s["rot"], ffn_hidden_size=s["ff"], vocab_size=VOCAB,
                       use_mla=True, q_lora_rank=0, kv_lora_rank=s["rank"], qk_nope_head_dim=s["dim"],
                       qk_rope_head_dim=s["rot"], v_head_dim=s["vdim"], num_experts=s["experts"], moe_top_k=s["top"],
                       moe_ffn_hidden_size=ff, moe_shared_expert_ffn=ff, first_k_dense=0, moe_layer_freq=2)


def active_weights(eng, s, n):
    """Weights a token is multiplied with, without the vocabulary matrices."""
    cfg = eng.cfg
    if eng.plan is None:
        return cfg.active_parameters() - 2 * cfg.vocab_size * cfg.hidden_size
    return cfg.num_parameters(include_embedding=False) - _idle_experts(s, s["top"])


def _idle_experts(s, used):
    """Weights of the routed experts beyond ``used`` per expert layer (about the same in the compared model)."""
    return (s["layers"] // 2) * (s["experts"] - used) * 2 * s["eff"] * s["width"]


def decode_bytes(kind, s, eng, B, ctx):
    """HBM bytes one decode step has to move: weights once (of the experts, those that B tokens choose at random), cached
    latents, recurrent state in and out."""
    cfg = eng.cfg
    hit = s["experts"] * (1 - (1 - s["top"] / s["experts"]) ** B)
    w = cfg.num_parameters(include_embedding=False) + cfg.vocab_size * cfg.hidden_size - _idle_experts(s, hit)
    n_lat = s["layers"] // 4 if kind == "kedesun" else s["layers"]
    cache = n_lat * B * (ctx + 1) * (s["rank"] + s["rot"]) * 2
    state = (s["layers"] - n_lat) * 2 * 4 * B * s["rh"] * s["rk"] * s["rv"]
    return 2 * w + cache + state


def kernel_table(s, prompts, length, B, ctx, bs=64):
    """[(phase, kernel, us, ideal us, like kernel, us, ideal us)]"""
    from ..models.layer_plan import LatentAttentionSpec, RotarySpec
    from ..models.parallel_decoder import LatentAttentionMixer
    from .serve_bench import _rows, graph_us, peaks
    dev = torch.device("cuda")
    hbm, flops, _ = peaks()
    ideal = lambda byts, fl=0.0: max(byts / hbm, fl / flops) * 1e6
    bf, f32 = dict(dtype=torch.bfloat16, device=dev), dict(dtype=torch.float32, device=dev)
    H, dim, rot, vdim, rank, width = s["heads"], s["dim"], s["rot"], s["vdim"], s["rank"], s["width"]
    spec = LatentAttentionSpec(H, dim, rot, vdim, rank, (dim + rot) ** -0.5, RotarySpec(rot, 10000.0))
    mix = LatentAttentionMixer(spec, width, 1e-6, torch.bfloat16, dev)
    ly = mix.layout
    mix.up_kv.normal_(0, rank ** -0.5)
    mix.gain.fill_(1.0)
    table = []
    # ---- prompt: steps of the latent attention
    rows, nb = _rows(prompts, length, 0, 0, bs, dev)
    T = prompts * length
    pairs = prompts * length * (length + 1) / 2
    projs = [torch.randn(T, mix.columns, **bf) for _ in range(2)]
    cache = torch.zeros(nb, bs, ly.row, **bf)
    context = torch.randn(T, ly.row, **bf)
    out = torch.empty(T, mix.out_columns, **bf)
    t = graph_us([lambda p=p: la._prep(p, ly, mix.gain, mix.turns, rows, cache, context) for p in projs])
    x, g = [torch.randn(T, rank, **bf) for _ in range(2)], torch.ones(rank, **bf)
    like = graph_us([lambda a=a: fused.rmsnorm(a, g, 1e-6) for a in x])
    table.append(("prefill", "latent_prep", t, ideal(T * (3 * ly.row + 2 * H * rot) * 2), "rmsnorm (latent)", like,
                  ideal(T * rank * 4)))
    kv = torch.randn(T, H * (dim + vdim), **bf)
    up, la_linear = mix.up_kv, la.linear_forward
    la.linear_forward = lambda *a: kv            # the attention kernel alone
    try:
        t = graph_us([lambda p=p: la._portions(p, ly, up, rows, cache, context, out, None) for p in projs])
    finally:
        la.linear_forward = la_linear
    fl = 2.0 * pairs * H * (dim + rot + vdim)
    qkv = [torch.randn(T, 2 * H * (dim + rot), **bf) for _ in range(2)]
    v = torch.randn(T, H, vdim, **bf)
    view = lambda a, i: a.view(T, 2, H, dim + rot)[:, i]
    like = graph_us([lambda a=a: attention.flash_attn_varlen(view(a, 0), view(a, 1), v, rows.cu, rows.cu, length, length,
                                                             causal=True) for a in qkv])
    table.append(("prefill", "latent attention (attn_fwd LAT)", t, ideal(T * H * (2 * dim + rot + 2 * vdim) * 2, fl),
                  "attn_fwd 192/128", like, ideal(T * H * (2 * dim + 2 * rot + 2 * vdim) * 2, fl)))
    del projs, qkv, v, kv, context, out
    # ---- prompt: retention
    rh, rk, rv = s["rh"], s["rk"], s["rv"]
    off = [0, rh * rk, 2 * rh * rk, 2 * rh * rk + rh * rv]
    ld = off[3] + rh * rv
    projs = [torch.randn(T, ld, **bf) for _ in range(2)]
    decay = torch.full((rh,), 0.99, **f32)
    o = torch.empty(T, rh, rv, **f32)
    st = mm.MemoryState.allocate(prompts, rh, rk, rv, dev)
    com = (rk ** -0.5, rh, rk, rv, rows, st, o)
    fl = T * rh * (4.0 * rk * rv + 128.0 * (rk + rv))
    chunk_ideal = ideal(T * rh * ((2 * rk + rv) * 2 + rv * 4), fl)
    t = graph_us([lambda p=p: mm._chunk(p, off[:3], None, None, 0.0, *com, decay) for p in projs])
    gates, gate_b = torch.randn(T, 2 * rh, **f32), torch.randn(2 * rh, **f32)
    like = graph_us([lambda p=p: mm._chunk(p, off[:3], gates, gate_b, 15.0, *com) for p in projs])
    table.append(("prefill", "retention chunk", t, chunk_ideal, "matrix_memory_chunk", like, chunk_ideal))
    y, gain = torch.empty(T, rh * rv, **bf), torch.ones(rh * rv, **f32)
    t = graph_us([lambda p=p: mm._output(o, p, off[3], None, rv, 1e-6, y) for p in projs])
    like = graph_us([lambda p=p: mm._output(o, p, off[3], gain, rv, 1e-6, y) for p in projs])
    table.append(("prefill", "retention output", t, ideal(T * rh * rv * 8), "memory_output", like, ideal(T * rh * rv * 8)))
    del projs, o, y, gates
    # ---- residual step, activations, experts: prompt and decode
    E, K, ff, eff = s["experts"], s["top"], s["ff"], s["eff"]
    for phase, n, cp in (("prefill", T, 2), ("decode", B, 8)):
        depth_n = s["layers"] // 2
        hist = torch.randn(depth_n + 2, n, width, **f32)
        x, avg, gain = torch.randn(n, width, **f32), torch.rand(depth_n + 1, **f32), torch.ones(width, **f32)
        ys = [torch.randn(n, width, **bf) for _ in range(cp)]
        gb = torch.ones(width, **bf)
        like = graph_us([lambda a=a, b=b: fused.rmsnorm(a, gb, 1e-6, b) for a, b in zip(ys, ys[1:] + ys[:1])])
        lid = ideal(n * width * 8)
        t = graph_us([lambda y=y: depth.add_layer(hist, depth_n, x, y, avg, width, 1e-6, x, gain) for y in ys])
        table.append((phase, f"depth_average ({depth_n} back)", t, ideal(n * width * (4 * depth_n + 16)), "rmsnorm + residual",
                      like, lid))
        er = torch.randn(n * K, width, **bf)
        dest = torch.randperm(n * K, device=dev).int().view(n, K)
        w = torch.rand(n, K, **f32)
        t = graph_us([lambda y=y: depth.add_layer(hist, depth_n, x, y, avg, width, 1e-6, x, gain, (er, dest, w)) for y in ys])
        table.append((phase, f"depth_average ({depth_n} back, {K} experts)", t, ideal(n * width * (4 * depth_n + 16 + 2 * K)),
                      "rmsnorm + residual", like, lid))
        del hist, er
        srcs, dst = [torch.randn(n, 2 * ff, **bf) for _ in range(cp)], torch.empty(n, ff + 4096, **bf)[:, 4096:]
        t = graph_us([lambda a=a: moe.activate(moe.SILU_GATE, a, ff, ff, dst) for a in srcs])
        like = graph_us([lambda a=a: fused.swiglu(a) for a in srcs])
        table.append((phase, "ffn_act (silu gate)", t, ideal(n * ff * 6), "swiglu", like, ideal(n * ff * 6)))
        del srcs, dst
        corr, counts = torch.zeros(E, **f32), torch.zeros(E, dtype=torch.int32, device=dev)
        router = torch.randn(E + 1, width, **bf)
        rw = router.float()[:E].contiguous()

        def pick(y):
            counts.zero_()
            _, (idx, _, place) = moe.route_tokens(y, router, E, K, corr, counts)
            return moe.expert_rows(y, counts, idx, place)

        def like_pick(y):
            idx, _ = route(torch.nn.functional.linear(y.float(), rw), None, None, K)
            dst_, _ = build_dispatch_plan(idx.reshape(-1), E)
            xp = torch.zeros(padded_rows_bound(n * K, E), width, **bf)
            return xp.index_copy(0, dst_, y[torch.arange(n, device=dev).repeat_interleave(K)])
        t, like = graph_us([lambda y=y: pick(y) for y in ys]), graph_us([lambda y=y: like_pick(y) for y in ys])
        i = ideal(n * width * 2 * (2 + K) + E * width * 2)
        table.append((phase, "logits + choice + expert rows", t, i, "logits + route + dispatch", like, i))
        xs, _, offs = pick(ys[0])
        n_w = max(2, math.ceil(3e8 / (E * eff * width * 2)))
        ups = [torch.randn(E, eff, width, **bf) for _ in range(n_w)]
        hit = int((counts > 0).sum())
        gid = ideal((hit * eff * width + n * K * (width + eff)) * 2, 2.0 * n * K * width * eff)
        t = graph_us([lambda u=u: moe.grouped(xs, u, offs) for u in ups])
        # the like model's segments: the worst-case buffer of its dispatch
        big = torch.zeros(padded_rows_bound(n * K, E), width, **bf)
        like = graph_us([lambda u=u: grouped_gemm(big, u, offs) for u in ups])
        table.append((phase, "grouped GEMM (up)", t, gid, "grouped GEMM", like, gid))
        del xs, ups, big, ys
        torch.cuda.empty_cache()
    # ---- decode: latent attention
    rows, nb = _rows(0, 0, ctx, B, bs, dev)
    n_c = max(2, math.ceil(3e8 / (B * (ctx + 1) * ly.row * 2)))
    proj = torch.randn(B, mix.columns, **bf)
    caches = [torch.randn(nb, bs, ly.row, **bf) for _ in range(n_c)]
    t = graph_us([lambda c=c: la._prep(proj, ly, mix.gain, mix.turns, rows, c, None) for c in caches])
    x = torch.randn(B, rank, **bf)
    like = graph_us([lambda: fused.rmsnorm(x, g, 1e-6)] * 8)
    table.append(("decode", "latent_prep", t, ideal(B * (2 * ly.row + 2 * H * rot) * 2), "rmsnorm (latent)", like,
                  ideal(B * rank * 4)))
    out = torch.empty(B, mix.out_columns, **bf)
    q_lat, q_rope = torch.randn(H, B, ly.row_rank, **bf), torch.randn(B, H, ly.row_rot, **bf)
    o_lat = torch.empty_like(q_lat)
    bmm, la._bmm = la._bmm, lambda a, b, out: out      # the attention kernel alone
    try:
        t = graph_us([lambda c=c: la._absorbed(proj, ly, mix.up_kv, rows, 0, B, c, out, None) for c in caches])
    finally:
        la._bmm = bmm
    like = graph_us([lambda c=c: attention.mla_paged_decode(q_lat.transpose(0, 1), q_rope, c, rows.tables, rows.ctx, ctx + 1,
                                                            spec.scale, out=o_lat.transpose(0, 1)) for c in caches])
    i = ideal(B * (ctx + 1) * ly.row * 2 + B * H * (2 * ly.row_rank + rot) * 2,
              2.0 * B * (ctx + 1) * H * (2 * ly.row_rank + ly.row_rot))
    table.append(("decode", "mla_paged_decode (gated, two terms)", t, i, "mla_paged_decode", like, i))
    del caches
    # ---- decode: retention
    n_s = max(2, math.ceil(3e8 / (B * rh * rk * rv * 4)))
    sts = [mm.MemoryState.allocate(B, rh, rk, rv, dev) for _ in range(n_s)]
    proj, y = torch.randn(B, ld, **bf), torch.empty(B, rh * rv, **bf)
    t = graph_us([lambda st=st: mm.retention(proj, *off, decay, rk ** -0.5, rh, rk, rv, rv, rows, st, 1e-6, y) for st in sts])
    h, gw, gain = torch.randn(B, width, **bf), torch.randn(2 * rh, width, **bf), torch.ones(rh * rv, **f32)
    like = graph_us([lambda st=st: mm.matrix_memory(proj, *off, h, gw, gate_b, 15.0, rk ** -0.5, rh, rk, rv, rv, rows, st,
                                                    gain, 1e-6) for st in sts])
    i = ideal(2 * B * rh * rk * rv * 4)
    table.append(("decode", "retention step", t, i, "matrix_memory step", like, i))
    return table

"""Latent attention over the rows of a serving step: a paged cache with one row ``[normed latent | rotated key part]`` per
token, shared by all heads (``csrc/latent_attention.cu``, ``csrc/attention_fwd.cu``, ``csrc/mla_decode.cu``).  Prompt portions
expand the context they see to per-head keys and values; single tokens work on the latent itself, with the up-projections
folded into query and output.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Dict

import torch

from . import _lib
from .gemm import linear_forward
from .rows import StepRows
from .window_attention import general_attention

LAUNCHES = {"latent_attention": 0}
MAX_ROW, MAX_ROT = 1024, 256
_SCRATCH: Dict[tuple, torch.Tensor] = {}


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


def cached_row(rank: int, rot: int):
    """(latent columns, rotated columns) a cached row stores: a geometry of the decode kernel if one is wide enough, else
    the sizes rounded up for the general kernel."""
    for cv, dr in ((128, 32), (256, 64), (512, 64)):
        if rank <= cv and rot <= dr:
            return cv, dr
    if up8(rank) + up8(rot) > MAX_ROW or rot > MAX_ROT:
        raise ValueError(f"cached rows of {rank} + {rot} are not supported (at most {MAX_ROW} together, {MAX_ROT} rotated)")
    return up8(rank), up8(rot)


@dataclass
class LatentLayout:
    """Columns of the packed projection (all multiples of 8) and sizes as stored.  Head h's query: ``dim`` unrotated columns
    at ``q + h * (dim + row_rot)``, then the rotated ones."""
    q: int
    down: int
    gate: int
    heads: int
    dim: int        # per head, padded
    vdim: int       # per head, padded
    rank: int       # true latent size
    row_rank: int   # latent columns of a cached row
    rot: int        # true rotated size
    row_rot: int    # rotated columns of a cached row
    scale: float
    magnitude: float
    eps: float
    window: int = 0      # positions a token sees, itself included; 0: all before it
    gate_cols: int = 1   # gate logits per head: one, or one per (padded) value column

    @property
    def row(self):
        return self.row_rank + self.row_rot


def rotation_turns(frequencies) -> torch.Tensor:
    """[pairs, 2] 32-bit: turns per position of every rotated pair as value and remainder."""
    t = torch.tensor(frequencies, dtype=torch.float64) / (2 * math.pi)
    return torch.stack([t.float(), (t - t.float().double()).float()], -1)


def _rotate(x, cos, sin):
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)


def _ref(proj, ly: LatentLayout, gain, turns, up_kv, rows: StepRows, cache, out, sinks=None):
    T, H, bs = proj.shape[0], ly.heads, cache.shape[1]
    p = proj.float()
    a = 2 * math.pi * rows.pos.double()[:, None] * turns.double().sum(-1)
    cos, sin = (torch.cos(a) * ly.magnitude).float(), (torch.sin(a) * ly.magnitude).float()
    c = p[:, ly.down:ly.down + ly.rank]
    row = torch.zeros(T, ly.row)
    row[:, :ly.rank] = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + ly.eps) * gain
    kr = ly.down + ly.row_rank
    row[:, ly.row_rank:ly.row_rank + ly.rot] = _rotate(p[:, kr:kr + ly.rot], cos, sin)
    flat, live = cache.view(-1, ly.row), rows.slots >= 0
    flat[rows.slots[live].long()] = row[live].to(cache.dtype)
    q = p[:, ly.q:ly.q + H * (ly.dim + ly.row_rot)].view(T, H, -1)
    qr = _rotate(q[..., ly.dim:ly.dim + ly.rot], cos[:, None], sin[:, None])
    uk, uv = up_kv[:H * ly.dim].float().view(H, ly.dim, -1), up_kv[H * ly.dim:].float().view(H, ly.vdim, -1)
    g = torch.sigmoid(p[:, ly.gate:ly.gate + H * ly.gate_cols].view(T, H, -1))
    for t in range(T):
        if rows.slots[t] < 0:
            out[t] = 0
            continue
        i = int(rows.pos[t])
        j = torch.arange(max(0, i - ly.window + 1) if ly.window else 0, i + 1)
        ctx = flat[rows.tables[rows.row_seq[t], j // bs].long() * bs + j % bs].float()
        lat, rot = ctx[:, :ly.row_rank], ctx[:, ly.row_rank:ly.row_rank + ly.rot]
        s = (torch.einsum("hd,hdc,nc->hn", q[t, :, :ly.dim], uk, lat) + qr[t] @ rot.T) * ly.scale
        w = torch.softmax(s if sinks is None else torch.cat([s, sinks[:, None]], 1), -1)[:, :len(j)]
        o = torch.einsum("hn,nc,hvc->hv", w, lat, uv) * g[t]
        out[t] = o.reshape(-1).to(out.dtype)
    return out


def _prep(proj, ly: LatentLayout, gain, turns, rows: StepRows, cache, context):
    ctx = rows.contexts[ly.window] if context is not None else None
    ptrs = (ctypes.c_void_p * 10)(*[t.data_ptr() if t is not None else None for t in
                                    (proj, gain, turns, rows.pos, rows.slots, cache, context, rows.row_seq,
                                     ctx.cu if ctx else None, ctx.start if ctx else None)])
    dims = (ctypes.c_int * 11)(proj.shape[0], rows.portion_rows if context is not None else 0, ly.q, ly.dim + ly.row_rot,
                               ly.dim, ly.down, ly.heads, ly.rank, ly.row_rank, ly.rot, ly.row_rot)
    LAUNCHES["latent_attention"] += 1
    _lib.check(_lib.kernels().gk_latent_prep(int(proj.dtype == torch.float32), ptrs, proj.stride(0), dims, float(ly.eps),
                                             float(ly.magnitude), _lib.stream_ptr()), "latent_prep")


def _portions(proj, ly: LatentLayout, up_kv, rows: StepRows, cache, context, out, sinks):
    """Prompt portions: the rest of the context from the cache, expansion, tcgen05 attention."""
    lib, n, ctx = _lib.kernels(), rows.n_portions, rows.contexts[ly.window]
    if ctx.max_before:
        LAUNCHES["latent_attention"] += 1
        _lib.check(lib.gk_latent_gather(_lib.ptr(cache), _lib.ptr(rows.tables), _lib.ptr(rows.first_pos), _lib.ptr(ctx.cu),
                                        _lib.ptr(ctx.start), _lib.ptr(context), n, rows.tables.shape[1], cache.shape[1],
                                        ly.row * context.element_size(), ctx.max_before, _lib.stream_ptr()), "latent_gather")
    kv = linear_forward(context[:, :ly.row_rank], up_kv)
    q, kr, gate = proj[:, ly.q:], context[:, ly.row_rank:], proj[:, ly.gate:]
    ptrs = (ctypes.c_void_p * 9)(*[t.data_ptr() if t is not None else None for t in
                                   (q, kv, kr, gate, out, rows.cu, ctx.cu, _lib.err_flag(proj.device), sinks)])
    lds = (ctypes.c_longlong * 5)(proj.stride(0), kv.stride(0), context.stride(0), proj.stride(0), out.stride(0))
    dims = (ctypes.c_int * 11)(n, rows.portion_rows, ctx.rows, ly.heads, ly.dim, up8(ly.rot), ly.vdim,
                               ly.dim + ly.row_rot, rows.max_portion, ly.window, ly.gate_cols)
    LAUNCHES["latent_attention"] += 1
    _lib.check(lib.gk_latent_prefill(ptrs, lds, dims, float(ly.scale), _lib.stream_ptr()), "latent_prefill")


def _bmm(a, b, out):
    """Head-batched product; 32-bit operands never in TF32."""
    if a.dtype != torch.float32:
        return torch.bmm(a, b, out=out)
    tf32 = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        return torch.bmm(a, b, out=out)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = tf32


def _decode_scratch(device, floats: int):
    # one buffer per size class, never replaced: captured graphs keep the address
    n = 1 << max(20, (floats - 1).bit_length())
    buf = _SCRATCH.get((device.index, n))
    if buf is None:
        buf = _SCRATCH[device.index, n] = torch.empty(n, dtype=torch.float32, device=device)
    return buf


def _absorbed(proj, ly: LatentLayout, up_kv, rows: StepRows, lo: int, hi: int, cache, out, sinks):
    """Rows ``lo .. hi`` on the latent itself: query times key up-projection, attention over the cached rows, value
    up-projection.  Single tokens in bf16 take the decode kernel, everything else the general one."""
    T, H = hi - lo, ly.heads
    p = proj[lo:hi]
    q = p[:, ly.q:ly.q + H * (ly.dim + ly.row_rot)].view(T, H, ly.dim + ly.row_rot)
    uk, uv = up_kv[:H * ly.dim].view(H, ly.dim, -1), up_kv[H * ly.dim:].view(H, ly.vdim, -1)
    kw = dict(dtype=proj.dtype, device=proj.device)
    lib = _lib.kernels()
    gate = p[:, ly.gate:]
    head_gate = gate if ly.gate_cols == 1 else None     # the attention kernels apply one per head themselves
    if lo == rows.portion_rows and proj.dtype == torch.bfloat16 and lib.gk_mla_decode_supported(ly.row_rank, ly.row_rot):
        q_lat = _bmm(q[..., :ly.dim].transpose(0, 1), uk, torch.empty(H, T, ly.row_rank, **kw))
        o_lat = torch.empty_like(q_lat)
        need = ctypes.c_longlong()
        span = min(ly.window, rows.max_ctx) if ly.window else rows.max_ctx
        lib.gk_mla_decode_scratch(T, H, ly.row_rank, span, ctypes.byref(need))
        scratch, tab = _decode_scratch(proj.device, max(need.value, 1)), rows.tables[rows.n_portions:]
        LAUNCHES["latent_attention"] += 1
        _lib.check(lib.gk_mla_paged_decode_gated(
            _lib.ptr(q_lat), q_lat.stride(1), q_lat.stride(0), _lib.ptr(q[..., ly.dim:]), q.stride(0), q.stride(1),
            _lib.ptr(cache), _lib.ptr(tab), _lib.ptr(rows.ctx), _lib.ptr(o_lat), o_lat.stride(1), o_lat.stride(0),
            _lib.ptr(scratch), T, H, ly.row_rank, ly.row_rot, cache.shape[1], rows.tables.shape[1], rows.max_ctx,
            float(ly.scale), _lib.ptr(head_gate), p.stride(0), ly.window, _lib.ptr(sinks), _lib.stream_ptr()),
            "mla_paged_decode_gated")
    else:
        q_abs, o = torch.empty(T, H, ly.row, **kw), torch.empty(T, H, ly.row_rank, **kw)
        q_abs[..., ly.row_rank:].copy_(q[..., ly.dim:])
        _bmm(q[..., :ly.dim].transpose(0, 1), uk, q_abs[..., :ly.row_rank].transpose(0, 1))
        general_attention(q_abs, H * ly.row, cache, rows, lo, hi, o, H, 1, ly.row, ly.scale, ly.row_rank,
                          ly.window, gate=head_gate, gate_ld=p.stride(0), sinks=sinks)
        o_lat = o.transpose(0, 1)
    _bmm(o_lat, uv.transpose(1, 2), out[lo:hi].view(T, H, ly.vdim).transpose(0, 1))
    if head_gate is None:
        LAUNCHES["latent_attention"] += 1
        _lib.check(lib.gk_gate_columns(int(proj.dtype == torch.float32), _lib.ptr(out[lo:hi]), out.stride(0), _lib.ptr(gate),
                                       p.stride(0), T, H * ly.vdim, _lib.stream_ptr()), "gate_columns")


def latent_attention(proj, ly: LatentLayout, gain, turns, up_kv, rows: StepRows, cache, out, sinks=None):
    """Appends every row's ``[latent | rotated key part]`` to ``cache`` [blocks, block_size, 1, row] and writes the gated
    attention output [T, heads * vdim] to ``out`` (any row stride).  The queries' rotated parts in ``proj`` are rotated in
    place.  ``up_kv`` [heads * (dim + vdim), row_rank]: key rows of all heads, then value rows; ``gain`` [rank] is
    32-bit, ``turns`` comes from ``rotation_turns``; ``sinks`` [heads] 32-bit join the softmax denominators."""
    cache = cache.view(cache.shape[0], cache.shape[1], ly.row)
    if not proj.is_cuda:
        return _ref(proj, ly, gain, turns, up_kv, rows, cache, out, sinks)
    T, P = proj.shape[0], rows.portion_rows
    tiled = P > 0 and proj.dtype == torch.bfloat16 and bool(
        _lib.kernels().gk_latent_prefill_supported(ly.dim, up8(ly.rot), ly.vdim))
    context = torch.empty(rows.contexts[ly.window].rows, ly.row, dtype=proj.dtype, device=proj.device) if tiled else None
    _prep(proj, ly, gain, turns, rows, cache, context)
    if tiled:
        _portions(proj, ly, up_kv, rows, cache, context, out, sinks)
    elif P:
        _absorbed(proj, ly, up_kv, rows, 0, P, cache, out, sinks)
    if T > P:
        _absorbed(proj, ly, up_kv, rows, P, T, cache, out, sinks)
    return out

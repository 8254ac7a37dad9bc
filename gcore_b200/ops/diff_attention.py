"""Differential attention over the rows of a serving step: heads subtract two causal softmax maps over the same values, and
the difference is normed, scaled and gated (``csrc/diff_attention.cu``, ``csrc/diff_prefill.cu``).  The paged cache holds one
row ``[two keys per kv head | one value per kv head]`` per token.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _lib
from .latent_attention import _rotate
from .rows import StepRows
from .window_attention import _decode_scratch, general_attention

LAUNCHES = {"diff_attention": 0}


@dataclass
class DiffLayout:
    """Columns of the packed projection (all multiples of 8) and sizes as stored: head h's queries at ``q + 2h * dim`` and
    ``dim`` behind, kv head g's keys likewise at ``k``, its value at ``v + g * vdim``, head h's gate at ``gate + h``."""
    q: int
    k: int
    v: int
    gate: int
    heads: int
    kv_heads: int
    dim: int         # per map, padded
    vdim: int        # per head, padded
    true_vdim: int   # values the norm's mean is taken over
    rot: int         # leading dimensions of a map that are rotated
    magnitude: float
    scale: float
    out_scale: float
    eps: float

    @property
    def value_offset(self):
        """Columns of a cached row in front of the values."""
        return 2 * self.kv_heads * self.dim

    @property
    def row(self):
        return self.value_offset + self.kv_heads * self.vdim


def _ref(proj, ly: DiffLayout, turns, lam, rows: StepRows, cache, out):
    T, H, G, bs = proj.shape[0], ly.heads, ly.kv_heads, cache.shape[1]
    p = proj.float()
    a = 2 * math.pi * rows.pos.double()[:, None, None] * turns.double().sum(-1)
    cos, sin = (torch.cos(a) * ly.magnitude).float(), (torch.sin(a) * ly.magnitude).float()
    q = p[:, ly.q:ly.q + 2 * H * ly.dim].view(T, 2 * H, ly.dim).clone()
    k = p[:, ly.k:ly.k + 2 * G * ly.dim].view(T, 2 * G, ly.dim).clone()
    for x in (q, k):
        x[..., :ly.rot] = _rotate(x[..., :ly.rot], cos, sin)
    row = torch.cat([k.flatten(1), p[:, ly.v:ly.v + G * ly.vdim]], 1)
    flat, live = cache.view(-1, ly.row), rows.slots >= 0
    flat[rows.slots[live].long()] = row[live].to(cache.dtype)
    gate = torch.sigmoid(p[:, ly.gate:ly.gate + H])
    for t in range(T):
        if rows.slots[t] < 0:
            out[t] = 0
            continue
        j = torch.arange(int(rows.pos[t]) + 1)
        ctx = flat[rows.tables[rows.row_seq[t], j // bs].long() * bs + j % bs].float()
        keys = ctx[:, :ly.value_offset].view(len(j), G, 2, ly.dim)
        vals = ctx[:, ly.value_offset:].view(len(j), G, ly.vdim)
        s = torch.einsum("grmd,ngmd->grmn", q[t].view(G, H // G, 2, ly.dim), keys) * ly.scale
        a = torch.einsum("grmn,ngv->grmv", torch.softmax(s, -1), vals)
        o = (a[:, :, 0] - lam * a[:, :, 1]).reshape(H, ly.vdim)
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / ly.true_vdim + ly.eps) * ly.out_scale * gate[t][:, None]
        out[t] = o.reshape(-1).to(out.dtype)
    return out


def _append(proj, ly: DiffLayout, turns, rows: StepRows, lo: int, hi: int, cache):
    """Rows ``lo .. hi``: queries rotated in place, rotated keys and the values to the cache."""
    ptrs = (ctypes.c_void_p * 5)(*[t.data_ptr() for t in (proj[lo:hi], turns, rows.pos[lo:hi], rows.slots[lo:hi], cache)])
    dims = (ctypes.c_int * 9)(hi - lo, ly.q, ly.k, ly.v, 2 * ly.heads, 2 * ly.kv_heads, ly.dim, ly.kv_heads * ly.vdim, ly.rot)
    LAUNCHES["diff_attention"] += 1
    _lib.check(_lib.kernels().gk_rotate_append(int(proj.dtype == torch.float32), ptrs, proj.stride(0), dims,
                                               float(ly.magnitude), _lib.stream_ptr()), "rotate_append")


def _finish(a, maps: int, proj, ly: DiffLayout, lam, out):
    """Heads from their maps (or, ``maps`` = 1, differences) in 32-bit rows."""
    ptrs = (ctypes.c_void_p * 4)(*[t.data_ptr() for t in (a, proj[:, ly.gate:], out, lam)])
    dims = (ctypes.c_int * 4)(proj.shape[0], ly.heads, ly.vdim, ly.true_vdim)
    LAUNCHES["diff_attention"] += 1
    _lib.check(_lib.kernels().gk_diff_combine(int(proj.dtype == torch.float32), maps, ptrs, proj.stride(0), out.stride(0), dims,
                                              (ctypes.c_float * 2)(ly.out_scale, ly.eps), _lib.stream_ptr()), "diff_combine")


def _general(proj, ly: DiffLayout, turns, lam, rows: StepRows, lo: int, hi: int, cache, out):
    """Any size, any dtype: both maps as heads of their own, then the difference."""
    _append(proj, ly, turns, rows, lo, hi, cache)
    p, H, G = proj[lo:hi], ly.heads, ly.kv_heads
    a = torch.empty(hi - lo, H, 2, ly.vdim, dtype=torch.float32, device=proj.device)
    general_attention(p[:, ly.q:], proj.stride(0), cache, rows, lo, hi, a, 2 * H, G, ly.dim, ly.scale, ly.vdim, maps=2,
                      v_off=ly.value_offset, v_stride=ly.vdim)
    _finish(a, 2, p, ly, lam, out[lo:hi])


def _portions(proj, ly: DiffLayout, turns, lam, rows: StepRows, cache, out):
    P, bs = rows.portion_rows, cache.shape[1]
    _append(proj, ly, turns, rows, 0, P, cache)
    wide = ly.vdim > 128
    diff = torch.empty(P, ly.heads, ly.vdim, dtype=torch.float32, device=proj.device) if wide else None
    ptrs = (ctypes.c_void_p * 10)(*[t.data_ptr() if t is not None else None for t in
                                    (proj[:, ly.q:], cache, rows.tables, rows.cu, rows.first_pos, proj[:, ly.gate:], out, lam,
                                     diff, _lib.err_flag(proj.device))])
    lds = (ctypes.c_longlong * 4)(proj.stride(0), proj.stride(0), out.stride(0), ly.row)
    dims = (ctypes.c_int * 12)(rows.n_portions, P, ly.heads, ly.kv_heads, ly.dim, ly.vdim, ly.true_vdim, ly.value_offset, bs,
                               rows.tables.shape[1], rows.max_portion, cache.shape[0])
    LAUNCHES["diff_attention"] += 1
    _lib.check(_lib.kernels().gk_diff_prefill(ptrs, lds, dims, (ctypes.c_float * 3)(ly.scale, ly.out_scale, ly.eps),
                                              _lib.stream_ptr()), "diff_prefill")
    if wide:
        _finish(diff, 1, proj[:P], ly, lam, out[:P])


def _decode(proj, ly: DiffLayout, turns, lam, rows: StepRows, cache, out):
    lib, P = _lib.kernels(), rows.portion_rows
    p, B = proj[P:], proj.shape[0] - P
    scratch = _decode_scratch(proj.device, max(1, int(lib.gk_diff_decode_scratch(B, ly.heads, ly.kv_heads, ly.vdim,
                                                                                 rows.max_ctx))))
    ptrs = (ctypes.c_void_p * 9)(*[t.data_ptr() for t in (p, cache, rows.tables[rows.n_portions:], rows.ctx, rows.slots[P:],
                                                          turns, lam, out[P:], scratch)])
    lds = (ctypes.c_longlong * 2)(proj.stride(0), out.stride(0))
    dims = (ctypes.c_int * 15)(B, ly.heads, ly.kv_heads, ly.dim, ly.vdim, ly.true_vdim, ly.rot, ly.q, ly.k, ly.v, ly.gate,
                               ly.row, cache.shape[1], rows.tables.shape[1], rows.max_ctx)
    LAUNCHES["diff_attention"] += 1
    _lib.check(lib.gk_diff_decode(ptrs, lds, dims, (ctypes.c_float * 4)(ly.scale, ly.magnitude, ly.out_scale, ly.eps),
                                  _lib.stream_ptr()), "diff_decode")


def differential_attention(proj, ly: DiffLayout, turns, lam, rows: StepRows, cache, out):
    """Appends every row's keys and values to ``cache`` [blocks, block_size, row] and writes the gated attention output
    [T, heads * vdim] to ``out`` (any row stride).  The queries in ``proj`` may be rotated in place.  ``turns`` comes from
    ``latent_attention.rotation_turns``; ``lam`` [1] 32-bit is the weight of the second map."""
    if not proj.is_cuda:
        return _ref(proj, ly, turns, lam, rows, cache, out)
    lib, T, P, bs = _lib.kernels(), proj.shape[0], rows.portion_rows, cache.shape[1]
    bf16 = proj.dtype == torch.bfloat16
    if P:
        if bf16 and (bs in (8, 16, 32) or bs % 64 == 0) and lib.gk_diff_prefill_supported(ly.dim, ly.vdim):
            _portions(proj, ly, turns, lam, rows, cache, out)
        else:
            _general(proj, ly, turns, lam, rows, 0, P, cache, out)
    if T > P:
        if bf16 and lib.gk_diff_decode_supported(ly.dim, ly.vdim):
            _decode(proj, ly, turns, lam, rows, cache, out)
        else:
            _general(proj, ly, turns, lam, rows, P, T, cache, out)
    return out

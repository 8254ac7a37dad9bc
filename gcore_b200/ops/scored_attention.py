"""Grouped-query attention with a bias on every score over the rows of a serving step (``csrc/scored_attention.cu``,
``csrc/scored_prefill.cu``): softmax weights with a logarithmic distance penalty over a sliding window and the first positions, or
sigmoid weights with a bias per head; queries and keys may be rotated and normed.  The paged cache holds one row
``[keys | values]`` per token.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from .head_prep import head_prep, rotate_heads, unit_heads
from .rows import StepRows
from .window_attention import _decode_scratch, append_keys, general_attention

LAUNCHES = {"scored_attention": 0}


@dataclass
class ScoredLayout:
    """Columns of the packed projection (all multiples of 8; the values follow the keys) and sizes as stored."""
    q: int
    k: int
    v: int
    heads: int
    kv_heads: int
    dim: int             # per head, padded
    true_dim: int        # dimensions of the norm's mean
    vdim: int            # per head, padded
    scale: float
    eps: float
    unit: bool = False   # queries and keys are divided by their root mean square
    sigmoid: bool = False
    window: int = 0
    keep: int = 0

    @property
    def value_offset(self):
        return self.kv_heads * self.dim

    @property
    def row(self):
        return self.kv_heads * (self.dim + self.vdim)


def _seen(i: int, ly: ScoredLayout):
    j = torch.arange(i + 1)
    return j[(i - j < ly.window) | (j < ly.keep)] if ly.window else j


def _ref(proj, ly: ScoredLayout, turns, distance, head_bias, rows: StepRows, cache, out, out_scale):
    T, H, G, bs = proj.shape[0], ly.heads, ly.kv_heads, cache.shape[1]
    p = proj.float()
    q, k = p[:, ly.q:ly.q + H * ly.dim].view(T, H, -1), p[:, ly.k:ly.k + G * ly.dim].view(T, G, -1)
    if turns is not None:
        q, k = (rotate_heads(x, turns, rows.pos) for x in (q, k))
    if ly.unit:
        q, k = (unit_heads(x, ly.true_dim, ly.eps) for x in (q, k))
    row = torch.cat([k.flatten(1), p[:, ly.v:ly.v + G * ly.vdim]], 1)
    flat, live = cache.view(-1, ly.row), rows.slots >= 0
    flat[rows.slots[live].long()] = row[live].to(cache.dtype)
    for t in range(T):
        if rows.slots[t] < 0:
            out[t] = 0
            continue
        i = int(rows.pos[t])
        j = _seen(i, ly)
        ctx = flat[rows.tables[rows.row_seq[t], j // bs].long() * bs + j % bs].float()
        keys, vals = ctx[:, :ly.value_offset].view(len(j), G, ly.dim), ctx[:, ly.value_offset:].view(len(j), G, ly.vdim)
        s = torch.einsum("grd,ngd->grn", q[t].view(G, H // G, ly.dim), keys).reshape(H, -1) * ly.scale
        if distance is not None:
            s = s - distance[0][:, None] * torch.log1p(distance[1][:, None] * (i - j).float())
        if head_bias is not None:
            s = s + head_bias[:, None]
        w = torch.sigmoid(s) if ly.sigmoid else torch.softmax(s, -1)
        o = torch.einsum("grn,ngv->grv", w.view(G, H // G, -1), vals) * out_scale
        out[t] = o.reshape(-1).to(out.dtype)
    return out


def _prepare(proj, ly: ScoredLayout, turns, rows: StepRows, lo: int, hi: int, cache):
    """Rows ``lo .. hi``: queries ready in place, keys and values in the cache."""
    if turns is None and not ly.unit:
        append_keys(proj[lo:hi], ly.k, ly.row, rows.slots[lo:hi], cache)
    else:
        head_prep(proj, rows, lo, hi, ly.q, ly.heads, ly.k, ly.kv_heads, ly.dim, turns, ly.true_dim if ly.unit else 0, ly.eps,
                  cache, ly.v, ly.kv_heads * ly.vdim)


def _general(proj, ly: ScoredLayout, turns, distance, head_bias, rows: StepRows, lo: int, hi: int, cache, out, out_scale):
    """Any size, any dtype."""
    _prepare(proj, ly, turns, rows, lo, hi, cache)
    general_attention(proj[lo:hi, ly.q:], proj.stride(0), cache, rows, lo, hi, out[lo:hi], ly.heads, ly.kv_heads, ly.dim, ly.scale,
                      ly.vdim, ly.window, v_off=ly.value_offset, v_stride=ly.vdim, keep=ly.keep, distance=distance,
                      head_bias=head_bias, sigmoid=ly.sigmoid, out_scale=out_scale)


def _ptrs(*tensors):
    return (ctypes.c_void_p * len(tensors))(*[t.data_ptr() if t is not None else None for t in tensors])


def _portions(proj, ly: ScoredLayout, turns, distance, head_bias, rows: StepRows, cache, out, out_scale):
    P, bs = rows.portion_rows, cache.shape[1]
    _prepare(proj, ly, turns, rows, 0, P, cache)
    r1, r2 = distance if distance is not None else (None, None)
    ptrs = _ptrs(proj[:, ly.q:], cache, rows.tables, rows.cu, rows.first_pos, r1, r2, head_bias, out, _lib.err_flag(proj.device))
    lds = (ctypes.c_longlong * 3)(proj.stride(0), out.stride(0), ly.row)
    dims = (ctypes.c_int * 13)(rows.n_portions, P, ly.heads, ly.kv_heads, ly.dim, ly.vdim, bs, rows.tables.shape[1],
                               rows.max_portion, cache.shape[0], ly.window, ly.keep, int(ly.sigmoid))
    LAUNCHES["scored_attention"] += 1
    _lib.check(_lib.kernels().gk_scored_prefill(ptrs, lds, dims, (ctypes.c_float * 2)(ly.scale, out_scale), _lib.stream_ptr()),
               "scored_prefill")


def _decode(proj, ly: ScoredLayout, turns, distance, head_bias, rows: StepRows, cache, out, out_scale):
    lib, P = _lib.kernels(), rows.portion_rows
    p, B = proj[P:], proj.shape[0] - P
    scratch = _decode_scratch(proj.device, max(1, int(lib.gk_scored_decode_scratch(B, ly.heads, ly.kv_heads, ly.vdim, ly.window,
                                                                                   ly.keep, rows.max_ctx))))
    r1, r2 = distance if distance is not None else (None, None)
    ptrs = _ptrs(p, cache, rows.tables[rows.n_portions:], rows.ctx, rows.slots[P:], turns, r1, r2, head_bias, out[P:], scratch)
    lds = (ctypes.c_longlong * 2)(proj.stride(0), out.stride(0))
    dims = (ctypes.c_int * 17)(B, ly.heads, ly.kv_heads, ly.dim, ly.vdim, 2 * turns.shape[0] if turns is not None else 0,
                               ly.true_dim if ly.unit else 0, ly.q, ly.k, ly.v, ly.row, cache.shape[1], rows.tables.shape[1],
                               rows.max_ctx, ly.window, ly.keep, int(ly.sigmoid))
    LAUNCHES["scored_attention"] += 1
    _lib.check(lib.gk_scored_decode(ptrs, lds, dims, (ctypes.c_float * 3)(ly.scale, out_scale, ly.eps), _lib.stream_ptr()),
               "scored_decode")


def scored_attention(proj, ly: ScoredLayout, rows: StepRows, cache, out, turns=None, distance=None, head_bias=None,
                     out_scale: float = 1.0):
    """Appends every row's keys and values to ``cache`` [blocks, block_size, row] and writes the attention output times
    ``out_scale`` [T, heads * vdim] to ``out`` (any row stride).  The queries in ``proj`` may be prepared in place.  ``turns``
    (``latent_attention.rotation_turns``): rotation, neighbours paired; ``distance`` = (r1, r2) and ``head_bias``: [heads]
    32-bit."""
    if not proj.is_cuda:
        return _ref(proj, ly, turns, distance, head_bias, rows, cache, out, out_scale)
    lib, T, P, bs = _lib.kernels(), proj.shape[0], rows.portion_rows, cache.shape[1]
    args = (proj, ly, turns, distance, head_bias, rows)
    # the tensor-core kernels know the penalty beside the softmax and the bias beside sigmoids (a softmax ignores it)
    bf16 = proj.dtype == torch.bfloat16 and (distance is None if ly.sigmoid else head_bias is None)
    if P:
        if bf16 and (bs in (8, 16, 32) or bs % 64 == 0) and lib.gk_scored_prefill_supported(ly.dim, ly.vdim):
            _portions(*args, cache, out, out_scale)
        else:
            _general(*args, 0, P, cache, out, out_scale)
    if T > P:
        if bf16 and lib.gk_scored_decode_supported(ly.dim, ly.vdim):
            _decode(*args, cache, out, out_scale)
        else:
            _general(*args, P, T, cache, out, out_scale)
    return out

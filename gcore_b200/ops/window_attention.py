"""Sliding-window attention with a linear distance penalty on a paged cache whose rows are key and value at once
(``csrc/window_attention.cu``, ``csrc/window_prefill.cu``).  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
from typing import Dict

import torch

from . import _lib
from .rows import StepRows

LAUNCHES = {"window_attention": 0}
MAX_HEAD_DIM = 512
_SCRATCH: Dict[tuple, torch.Tensor] = {}


def padded_head_dim(dim: int) -> int:
    """Head size the kernels store: the tensor-core kernels are built for 64 and 128, larger heads run the general
    kernel (zero columns change neither scores nor outputs)."""
    if dim > MAX_HEAD_DIM:
        raise ValueError(f"attention heads of {dim} are not supported (at most {MAX_HEAD_DIM})")
    return 64 if dim <= 64 else 128 if dim <= 128 else (dim + 7) // 8 * 8


def _ref(proj, q_off, k_off, H, G, D, rows, cache, slopes, scale, window):
    bs = cache.shape[1]
    out = torch.zeros(proj.shape[0], H, D, dtype=proj.dtype)
    flat = cache.view(-1, G, D)
    live = rows.slots >= 0
    flat[rows.slots[live].long()] = proj[live, k_off:k_off + G * D].view(-1, G, D)
    for t in range(proj.shape[0]):
        if rows.slots[t] < 0:
            continue
        i = int(rows.pos[t])
        j = torch.arange(max(0, i - window + 1), i + 1)
        slots = rows.tables[rows.row_seq[t], j // bs].long() * bs + j % bs
        k = flat[slots].float().repeat_interleave(H // G, 1)                       # [n, H, D]
        s = torch.einsum("hd,nhd->hn", proj[t, q_off:q_off + H * D].view(H, D).float(), k) * scale
        p = torch.softmax(s - slopes[:, None] * (i - j).float()[None], -1)
        out[t] = torch.einsum("hn,nhd->hd", p, k).to(proj.dtype)
    return out.view(-1, H * D)


def _decode_scratch(device, floats: int):
    # one buffer per size class, never replaced: captured graphs keep the address
    n = 1 << max(20, (floats - 1).bit_length())
    buf = _SCRATCH.get((device.index, n))
    if buf is None:
        buf = _SCRATCH[device.index, n] = torch.empty(n, dtype=torch.float32, device=device)
    return buf


def append_keys(proj, k_off, n, slots, cache):
    """Copies ``n`` key elements at column ``k_off`` of every row to its cache slot."""
    es = proj.element_size()
    LAUNCHES["window_attention"] += 1
    _lib.check(_lib.kernels().gk_append_keys(_lib.ptr(proj), proj.stride(0) * es, k_off * es, n * es, _lib.ptr(slots),
                                             _lib.ptr(cache), slots.numel(), _lib.stream_ptr()), "append_keys")


def general_attention(q, q_ld, cache, rows: StepRows, lo, hi, out, H, G, D, scale, dv=None, window=0, slopes=None, gate=None,
                      gate_ld=0, sinks=None, maps=1, v_off=0, v_stride=None, keep=0, distance=None, head_bias=None,
                      sigmoid=False, out_scale=1.0):
    """Rows ``lo .. hi`` of a step against the paged cache, whose rows hold G * ``maps`` keys of ``D`` columns and, at
    ``v_off``, G values of ``dv`` columns ``v_stride`` apart (default: a value is the first columns of its key).  Optional
    window (0: none) beside the first ``keep`` positions, penalties (``slopes`` times the distance; ``distance`` = (r1, r2):
    r1 ln(1 + r2 distance)), bias per head, sink logits and output gate; ``sigmoid``: sigmoids of the scores in place of the
    softmax.  Any size, 32-bit or bf16; ``out`` [rows, H * dv] or [rows, H, ...] (any row stride) may be 32-bit."""
    row = cache.stride(1)
    dims = (ctypes.c_int * 13)(hi - lo, H, G, maps, D, dv or D, v_off, D if v_stride is None else v_stride, window,
                               cache.shape[1], rows.tables.shape[1], keep, int(sigmoid))
    r1, r2 = distance if distance is not None else (None, None)
    ptrs = (ctypes.c_void_p * 13)(*[t.data_ptr() if t is not None else None for t in
                                    (q, cache, rows.tables, rows.row_seq[lo:hi], rows.pos[lo:hi], rows.slots[lo:hi], slopes,
                                     gate, out, sinks, r1, r2, head_bias)])
    lds = (ctypes.c_longlong * 4)(q_ld, gate_ld, row, H * (dv or D) if out.dim() > 2 else out.stride(0))
    LAUNCHES["window_attention"] += 1
    _lib.check(_lib.kernels().gk_window_attn(int(q.dtype == torch.float32), int(out.dtype == torch.float32), ptrs, lds, dims,
                                             (ctypes.c_float * 2)(scale, out_scale), _lib.stream_ptr()), "window_attn")


def window_attention(proj, q_off: int, k_off: int, heads: int, kv_heads: int, dim: int, rows: StepRows, cache, slopes,
                     scale: float, window: int):
    """``proj`` [T, ld]: packed projections with the queries at ``q_off`` and the keys at ``k_off``.  Stores the new keys
    in ``cache`` [blocks, block_size, kv_heads, dim] and returns the attention output [T, heads * dim]."""
    H, G, D = heads, kv_heads, dim
    if not proj.is_cuda:
        return _ref(proj, q_off, k_off, H, G, D, rows, cache, slopes, scale, window)
    T, P, bs = proj.shape[0], rows.portion_rows, cache.shape[1]
    out = torch.empty(T, H * D, dtype=proj.dtype, device=proj.device)
    lib, bf16 = _lib.kernels(), proj.dtype == torch.bfloat16
    tiled = bf16 and D in (64, 128)
    if not tiled:
        append_keys(proj, k_off, G * D, rows.slots, cache)
        general_attention(proj[:, q_off:], proj.stride(0), cache, rows, 0, T, out, H, G, D, scale, None, window, slopes)
        return out
    if P:
        append_keys(proj[:P], k_off, G * D, rows.slots[:P], cache)
        if bs in (8, 16, 32) or bs % 64 == 0:
            dims = (ctypes.c_int * 12)(rows.n_portions, P, H, G, D, window, bs, rows.tables.shape[1], rows.max_portion,
                                       q_off, cache.shape[0], 0)
            LAUNCHES["window_attention"] += 1
            _lib.check(lib.gk_window_prefill(_lib.ptr(proj), proj.stride(0), _lib.ptr(cache), _lib.ptr(rows.tables),
                                             _lib.ptr(rows.cu), _lib.ptr(rows.first_pos), _lib.ptr(slopes),
                                             _lib.ptr(out), dims, float(scale), _lib.ptr(_lib.err_flag(proj.device)),
                                             _lib.stream_ptr()), "window_prefill")
        else:
            general_attention(proj[:, q_off:], proj.stride(0), cache, rows, 0, P, out, H, G, D, scale, None, window, slopes)
    if T > P:
        B = T - P
        ptab = rows.tables[rows.n_portions:]
        span = min(window, rows.max_ctx)
        scratch = _decode_scratch(proj.device, int(lib.gk_shared_kv_decode_scratch(B, H, D, span)))
        dims = (ctypes.c_int * 10)(B, H, G, D, window, bs, rows.tables.shape[1], rows.max_ctx, q_off, k_off)
        LAUNCHES["window_attention"] += 1
        _lib.check(lib.gk_shared_kv_decode(_lib.ptr(proj[P:]), proj.stride(0), _lib.ptr(cache), _lib.ptr(ptab),
                                           _lib.ptr(rows.ctx), _lib.ptr(rows.slots[P:]), _lib.ptr(slopes),
                                           _lib.ptr(out[P:]), _lib.ptr(scratch), dims, float(scale),
                                           _lib.stream_ptr()), "shared_kv_decode")
    return out

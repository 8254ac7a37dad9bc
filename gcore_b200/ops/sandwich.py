"""Residual-stream steps of decoders with norms before and after every sublayer and a 32-bit residual
(``csrc/sandwich_norm.cu``).  Each call takes a sublayer's output to the next sublayer's input in one launch.  Gains are
32-bit vectors; a gain stored around zero is passed as ``1 + w``.  Rows may be padded with zero columns: ``width`` is the
count the means are taken over.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

LAUNCHES = {"sandwich": 0}
_EMBED, _ONE, _PAIR, _ROWS = 0, 1, 2, 3


def _rms(x, width, eps):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / width + eps)


def _launch(src, like, x, n_rows, width, eps, vocab=0, max_pos=0, **t):
    names = ("tokens", "pos", "embed", "pos_table", "ya", "yb", "gain_a", "gain_b", "gain_post", "x", "x_first", "x_add",
             "step", "rows", "gain_pre", "h")
    t["x"] = x
    for k in ("embed", "pos_table", "ya", "yb", "gain_a", "gain_b", "gain_post", "x", "x_add", "step", "gain_pre"):
        assert t.get(k) is None or t[k].is_contiguous(), k
    ptrs = (ctypes.c_void_p * len(names))(*[t[k].data_ptr() if t.get(k) is not None else None for k in names])
    dims = (ctypes.c_int * 5)(vocab, max_pos, n_rows, x.shape[1], width)
    LAUNCHES["sandwich"] += 1
    _lib.check(_lib.kernels().gk_sandwich_norm(src, int(like == torch.float32), ptrs, dims, float(eps),
                                               _lib.stream_ptr()), "sandwich_norm")


def embed_rows(tokens, pos, embed, pos_table, gain_pre, width, eps, step=None, keep_first=False, x=None):
    """``x = embed[token] + pos_table[pos]`` (kept as ``first`` when asked), ``+ step``; returns ``(x, first, h)`` with
    ``h`` the normed input of the first sublayer.  ``tokens`` int64, ``pos`` int32; ``pos_table`` None: tokens alone; ``x``: where the
    stream goes."""
    T, H = tokens.numel(), embed.shape[1]
    if not embed.is_cuda:
        first = embed[tokens].float()
        if pos_table is not None:
            first = first + pos_table[pos.long()].float()
        first_x = first + step if step is not None else first.clone()
        x = first_x if x is None else x.copy_(first_x)
        return x, (first if keep_first else None), (_rms(x, width, eps) * gain_pre).to(embed.dtype)
    x = torch.empty(T, H, dtype=torch.float32, device=embed.device) if x is None else x
    first = torch.empty_like(x) if keep_first else None
    h = torch.empty(T, H, dtype=embed.dtype, device=embed.device)
    _launch(_EMBED, embed.dtype, x, T, width, eps, embed.shape[0], 0 if pos_table is None else pos_table.shape[0],
            tokens=tokens, pos=pos, embed=embed, pos_table=pos_table, x_first=first, step=step, gain_pre=gain_pre, h=h)
    return x, first, h


def add_sublayer(x, y, gain_post, width, eps, gain_pre=None, x_add=None, step=None, y2=None, gain_a=None, gain_b=None):
    """``x += norm(m) * gain_post [+ x_add] [+ step]`` in place, with ``m = y`` or, for two mixers side by side,
    ``m = (norm(y) * gain_a + norm(y2) * gain_b) / 2``.  Returns ``norm(x) * gain_pre`` in ``y``'s dtype (None without
    ``gain_pre``)."""
    if not y.is_cuda:
        m = y.float()
        if y2 is not None:
            m = 0.5 * (_rms(m, width, eps) * gain_a + _rms(y2.float(), width, eps) * gain_b)
        x += _rms(m, width, eps) * gain_post
        if x_add is not None:
            x += x_add
        if step is not None:
            x += step
        return (_rms(x, width, eps) * gain_pre).to(y.dtype) if gain_pre is not None else None
    h = torch.empty_like(y) if gain_pre is not None else None
    _launch(_PAIR if y2 is not None else _ONE, y.dtype, x, x.shape[0], width, eps, ya=y, yb=y2, gain_a=gain_a,
            gain_b=gain_b, gain_post=gain_post, x_add=x_add, step=step, gain_pre=gain_pre, h=h)
    return h


def norm_rows(x, gain, width, eps, dtype, rows=None):
    """``norm(x[rows]) * gain`` of the 32-bit residual, in ``dtype``."""
    if not x.is_cuda:
        src = x if rows is None else x[rows]
        return (_rms(src, width, eps) * gain).to(dtype)
    n = x.shape[0] if rows is None else rows.numel()
    h = torch.empty(n, x.shape[1], dtype=dtype, device=x.device)
    _launch(_ROWS, dtype, x, n, width, eps, rows=rows, gain_pre=gain, h=h)
    return h


def swiglu(x):
    """``silu(x[:, :F]) * x[:, F:]``: the framework's kernel in bf16, a true 32-bit one for 32-bit rows."""
    from . import fused
    if x.is_cuda and x.dtype == torch.float32:
        T, F = x.shape[0], x.shape[1] // 2
        out = torch.empty(T, F, dtype=x.dtype, device=x.device)
        LAUNCHES["sandwich"] += 1
        _lib.check(_lib.kernels().gk_swiglu_f32(_lib.ptr(x), _lib.ptr(out), T, F, _lib.stream_ptr()), "swiglu_f32")
        return out
    return fused.swiglu(x)

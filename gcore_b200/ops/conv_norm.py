"""Residual steps of pre-norm decoders whose sublayers read their normed input through a short causal convolution over time
(``csrc/conv_norm.cu``): a sublayer's output joins the 32-bit residual, the sum is normed, and every channel becomes
``sum_j w[j] * h[t - taps + 1 + j]``, all in one launch.  A request keeps its last ``taps - 1`` normed inputs in 32-bit, the one
of position p in ring row ``p mod (taps - 1)``.  Rows may be padded with zero columns: ``width`` is the count the means are
taken over.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .rows import StepRows

LAUNCHES = {"conv_norm": 0}
MAX_TAPS, MAX_WIDTH = 16, 16384
STORED_TAPS = (2, 3, 4, 8, 16)      # taps the kernel is built for; others are padded with zero taps in front


def stored_taps(taps: int) -> int:
    if not 1 <= taps <= MAX_TAPS:
        raise ValueError(f"input convolutions of 1 to {MAX_TAPS} taps are supported, not {taps}")
    return next(n for n in STORED_TAPS if n >= taps)


@dataclass
class NormSpec:
    """Norm in front of a sublayer: over ``width`` columns, with the mean taken off first (``center``) or not."""
    width: int
    eps: float
    center: bool = True


def norm(x, gain, spec: NormSpec):
    """32-bit rows, normed."""
    if spec.center:
        d = x - x[:, :spec.width].mean(-1, keepdim=True)
        d[:, spec.width:] = 0
    else:
        d = x
    return d * torch.rsqrt(d.pow(2).sum(-1, keepdim=True) / spec.width + spec.eps) * gain


def _convolve(h, taps, ring, rows: StepRows):
    """``taps`` [n, H], ``ring`` [slots, n - 1, H]: state of every request slot."""
    n, out = taps.shape[0], torch.empty_like(h)
    cu = [0] if rows.cu is None else rows.cu.tolist()
    edges = cu + list(range(cu[-1] + 1, h.shape[0] + 1))
    for s, (lo, hi) in enumerate(zip(edges, edges[1:])):
        slot, p0 = int(rows.states[s]), int(rows.first_pos[s])
        past = [ring[slot, p % (n - 1)].clone() if p >= 0 and slot >= 0 else torch.zeros_like(h[0]) for p in range(p0 - n + 1, p0)]
        seq = torch.stack(past + list(h[lo:hi]))
        for t in range(hi - lo):
            out[lo + t] = (taps * seq[t:t + n]).sum(0)
        if slot >= 0:
            for t in range(max(0, hi - lo - n + 1), hi - lo):
                ring[slot, (p0 + t) % (n - 1)] = h[lo + t]
    return out


def _launch(rows: Optional[StepRows], n_rows: int, H: int, spec: NormSpec, mult: float, vocab: int, n_taps: int, fp32: bool, **t):
    names = ("tokens", "embed", "x", "y", "x_out", "gain", "taps", "ring", "cu", "first_pos", "states", "pick", "h")
    if n_taps:
        t.update(cu=rows.cu, first_pos=rows.first_pos, states=rows.states)
    for k in names:
        assert t.get(k) is None or t[k].is_contiguous(), k
    ptrs = (ctypes.c_void_p * len(names))(*[t[k].data_ptr() if t.get(k) is not None else None for k in names])
    portions = (rows.n_portions, rows.portion_rows, rows.max_portion) if n_taps else (0, 0, 0)
    dims = (ctypes.c_int * 9)(n_rows, H, spec.width, *portions, n_taps, vocab, int(spec.center))
    floats = (ctypes.c_float * 2)(mult, spec.eps)
    LAUNCHES["conv_norm"] += 1
    _lib.check(_lib.kernels().gk_conv_norm(int(fp32), ptrs, dims, floats, _lib.stream_ptr()), "conv_norm")


def conv_embed_rows(rows: StepRows, embed, gain, taps, ring, spec: NormSpec):
    """``x = embed[token]``; returns ``(x, h)`` with ``h`` the convolved norm of ``x``, the input of the first sublayer."""
    T, H = rows.tokens.numel(), embed.shape[1]
    if not embed.is_cuda:
        x = embed[rows.tokens].float()
        return x, _convolve(norm(x, gain, spec), taps, ring, rows).to(embed.dtype)
    x = torch.empty(T, H, dtype=torch.float32, device=embed.device)
    h = torch.empty(T, H, dtype=embed.dtype, device=embed.device)
    _launch(rows, T, H, spec, 0.0, embed.shape[0], taps.shape[0], embed.dtype == torch.float32, tokens=rows.tokens, embed=embed,
            x_out=x, gain=gain, taps=taps, ring=ring, h=h)
    return x, h


def conv_add_sublayer(x, y, mult: float, spec: NormSpec, gain=None, rows: Optional[StepRows] = None, taps=None, ring=None,
                 keep: bool = True):
    """``x + mult * y`` and, with ``gain``, its norm in ``y``'s dtype, convolved when ``taps`` are given.  Returns
    ``(x_new, h)``; ``x`` stays as it is (a row of ``h`` reads its neighbours), and without ``keep`` ``x_new`` is None."""
    if not y.is_cuda:
        new = x + mult * y.float()
        h = norm(new, gain, spec) if gain is not None else None
        if taps is not None:
            h = _convolve(h, taps, ring, rows)
        return (new if keep else None), (h.to(y.dtype) if h is not None else None)
    new = torch.empty_like(x) if keep else None
    h = torch.empty_like(y) if gain is not None else None
    _launch(rows, x.shape[0], x.shape[1], spec, mult, 0, taps.shape[0] if taps is not None else 0, y.dtype == torch.float32, x=x,
            y=y, x_out=new, gain=gain, taps=taps, ring=ring, h=h)
    return new, h


def conv_norm_rows(x, gain, spec: NormSpec, dtype, pick=None):
    """``norm(x[pick]) * gain`` of the 32-bit residual, in ``dtype``."""
    if not x.is_cuda:
        return norm(x if pick is None else x[pick], gain, spec).to(dtype)
    n = x.shape[0] if pick is None else pick.numel()
    h = torch.empty(n, x.shape[1], dtype=dtype, device=x.device)
    _launch(None, n, x.shape[1], spec, 0.0, 0, 0, dtype == torch.float32, x=x, gain=gain, pick=pick, h=h)
    return h

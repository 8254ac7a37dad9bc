"""Residual step of decoders that hand on a weighted average over depth (``csrc/depth_average.cu``): a layer's combined
update, the average over the embedding output and every layer's result so far, and the next layer's norm in one launch.
CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

LAUNCHES = {"depth": 0}


def add_layer(history, n: int, x_in, y, avg, width: int, eps: float, x_out, gain=None, routed=None, keep: bool = True):
    """``X_n = x_in + y [+ routed]`` (stored as ``history[n]`` if ``keep``), ``x_out = sum_{j <= n} avg[j] * X_j``; returns
    ``norm(x_out) * gain`` in ``y``'s dtype (None without ``gain``).  ``history`` [slots, T, H] 32-bit with X_0 .. X_(n-1);
    ``routed`` = (expert rows, dest [T, K] int32, weight [T, K]): the rows are weighted and added.  Rows may be padded with
    zero columns: ``width`` is the count the mean is taken over.  ``x_in`` may be ``x_out``."""
    T, H = y.shape
    if not y.is_cuda:
        new = x_in + y.float()
        if routed is not None:
            rows, dest, weight = routed
            new = new + (rows[dest.long()].float() * weight[:, :, None]).sum(1)
        out = avg[n] * new
        for j in range(n):
            out = out + avg[j] * history[j]
        if keep:
            history[n].copy_(new)
        x_out.copy_(out)
        if gain is None:
            return None
        return (out * torch.rsqrt(out.pow(2).sum(-1, keepdim=True) / width + eps) * gain).to(y.dtype)
    h = torch.empty_like(y) if gain is not None else None
    rows, dest, weight = routed if routed is not None else (None, None, None)
    for t in (x_in, x_out, y, history, rows, dest, weight):
        assert t is None or t.is_contiguous()
    ptrs = (ctypes.c_void_p * 11)(*[t.data_ptr() if t is not None else None for t in
                                    (x_in, y, rows, dest, weight, history, history[n] if keep else None, avg, x_out, gain,
                                     h)])
    dims = (ctypes.c_int * 5)(T, H, width, n, dest.shape[1] if dest is not None else 0)
    LAUNCHES["depth"] += 1
    _lib.check(_lib.kernels().gk_depth_average(int(y.dtype == torch.float32), ptrs, history.stride(0), dims, float(eps),
                                               _lib.stream_ptr()), "depth_average")
    return h

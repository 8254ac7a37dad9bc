"""Residual streams of decoders with hyper-connections (``csrc/stream_mix.cu``): the write of one sublayer, the mixture of the
streams, and the read and norm in front of the next sublayer in one launch.  The streams [T, S, H] are 32-bit.  CPU tensors
run the plain PyTorch definition."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

LAUNCHES = {"streams": 0}
MAX_STREAMS = 16


def _norm(u, gain, width, eps, dtype):
    return (u * torch.rsqrt(u.pow(2).sum(-1, keepdim=True) / width + eps) * gain).to(dtype)


def _launch(x, like, width, eps, vocab=0, keep=True, **t):
    names = ("tokens", "embed", "y", "routed", "dest", "weight", "mix", "write", "read", "gain", "h", "total")
    for n in names + ("x",):
        v = x if n == "x" else t.get(n)
        assert v is None or v.is_contiguous(), n
    ptrs = (ctypes.c_void_p * (len(names) + 1))(x.data_ptr(), *[t[n].data_ptr() if t.get(n) is not None else None
                                                                 for n in names])
    T, S, H = x.shape
    dest = t.get("dest")
    dims = (ctypes.c_int * 7)(T, S, H, width, dest.shape[1] if dest is not None else 0, vocab, int(keep))
    LAUNCHES["streams"] += 1
    _lib.check(_lib.kernels().gk_stream_mix(int(like == torch.float32), ptrs, dims, float(eps), _lib.stream_ptr()),
               "stream_mix")


def embed_rows(tokens, embed, streams: int, read, gain, width: int, eps: float):
    """All streams equal to ``embed[token]``; returns ``(x [T, S, H], h)`` with ``h = norm(sum_s read[s] x_s) * gain``."""
    T, H = tokens.numel(), embed.shape[1]
    if not embed.is_cuda:
        x = embed[tokens].float()[:, None].repeat(1, streams, 1)
        return x, _norm(torch.einsum("s,tsh->th", read, x), gain, width, eps, embed.dtype)
    x = torch.empty(T, streams, H, dtype=torch.float32, device=embed.device)
    h = torch.empty(T, H, dtype=embed.dtype, device=embed.device)
    if T:
        _launch(x, embed.dtype, width, eps, embed.shape[0], tokens=tokens, embed=embed, read=read, gain=gain, h=h)
    return x, h


def connect(x, y, mix, write, width: int, eps: float, read=None, gain=None, routed=None, total=None, keep=True):
    """``x_t <- sum_s mix[s, t] x_s + write[t] * (y + routed)``, all streams at once and in place (with ``keep``); then
    ``u = sum_s read[s] x_s`` (without ``read``: the streams' sum).  Returns ``norm(u) * gain`` in the sublayers' dtype
    (None without ``gain``) and stores ``u`` in ``total`` if given.  ``y`` may be None; ``routed`` = (expert rows,
    dest [T, K] int32, weight [T, K]): the rows are weighted and added."""
    dtype = y.dtype if y is not None else routed[0].dtype
    rows, dest, weight = routed if routed is not None else (None, None, None)
    if not x.is_cuda:
        add = y.float() if y is not None else 0
        if routed is not None:
            add = add + (rows[dest.long()].float() * weight[:, :, None]).sum(1)
        new = torch.einsum("st,nsh->nth", mix, x) + write[None, :, None] * add[:, None]
        u = new.sum(1) if read is None else torch.einsum("s,tsh->th", read, new)
        if keep:
            x.copy_(new)
        if total is not None:
            total.copy_(u)
        return _norm(u, gain, width, eps, dtype) if gain is not None else None
    h = torch.empty(x.shape[0], x.shape[2], dtype=dtype, device=x.device) if gain is not None else None
    if x.shape[0]:
        _launch(x, dtype, width, eps, keep=keep, y=y, routed=rows, dest=dest, weight=weight, mix=mix, write=write, read=read,
                gain=gain, h=h, total=total)
    return h

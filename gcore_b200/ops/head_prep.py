"""Heads of a packed projection made ready for a mixer (``csrc/scored_attention.cu``): rotation, division by the root mean square,
silu, and the append of keys and values to a paged cache.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
import math

import torch

from . import _lib
from .latent_attention import _rotate
from .rows import StepRows

LAUNCHES = {"head_prep": 0}


def rotate_heads(x, turns, pos):
    """``x`` [T, heads, dim] with its leading dimensions rotated, neighbours paired."""
    a = 2 * math.pi * pos.double()[:, None, None] * turns.double().sum(-1)
    n = 2 * turns.shape[0]
    return torch.cat([_rotate(x[..., :n], torch.cos(a).float(), torch.sin(a).float()), x[..., n:]], -1)


def unit_heads(x, true_dim: int, eps: float):
    """``x`` [..., dim] divided by its root mean square over ``true_dim`` dimensions (the others are zero)."""
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / true_dim + eps)


def head_prep(proj, rows: StepRows, lo: int, hi: int, q_off: int, q_heads: int, k_off: int, k_heads: int, dim: int, turns=None,
              unit_dim: int = 0, eps: float = 0.0, cache=None, v_off: int = 0, v_cols: int = 0):
    """Rows ``lo .. hi``: ``q_heads`` queries and ``k_heads`` keys of ``dim`` columns rotated (``turns``) and normed over
    ``unit_dim`` dimensions (0: not), queries in place; keys and ``v_cols`` value columns go to ``cache`` (rows of
    ``k_heads * dim + v_cols``), without one the keys stay in place too.  GPU tensors only."""
    ptrs = (ctypes.c_void_p * 5)(*[t.data_ptr() if t is not None else None for t in
                                   (proj[lo:hi], turns, rows.pos[lo:hi], rows.slots[lo:hi], cache)])
    dims = (ctypes.c_int * 10)(hi - lo, q_off, k_off, v_off, q_heads, k_heads, dim, v_cols,
                               2 * turns.shape[0] if turns is not None else 0, unit_dim)
    LAUNCHES["head_prep"] += 1
    _lib.check(_lib.kernels().gk_head_prep(int(proj.dtype == torch.float32), ptrs, proj.stride(0), dims, float(eps),
                                           _lib.stream_ptr()), "head_prep")


def silu_columns(proj, off: int, n: int):
    """Columns ``off .. off + n`` of ``proj`` become their silu."""
    if not proj.is_cuda:
        proj[:, off:off + n] = torch.nn.functional.silu(proj[:, off:off + n].float()).to(proj.dtype)
        return
    LAUNCHES["head_prep"] += 1
    _lib.check(_lib.kernels().gk_silu_columns(int(proj.dtype == torch.float32), _lib.ptr(proj), proj.stride(0), off, n,
                                              proj.shape[0], _lib.stream_ptr()), "silu_columns")

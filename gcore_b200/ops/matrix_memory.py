"""Recurrent matrix memories over the rows of a serving step (``csrc/matrix_memory.cu``, ``csrc/matrix_memory_chunk.cu``): the
gated memory of an mLSTM, and retention, whose decay is fixed per head (with a norm per head and a silu gate, or a joint norm and
a sigmoid gate, and with rotated or activated inputs).  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .gemm import linear_forward
from .head_prep import head_prep, rotate_heads, silu_columns
from .rows import StepRows

LAUNCHES = {"matrix_memory": 0}
SLICE = 64        # value columns per state slice (csrc/matrix_memory.cu: MM_SLICE)
MAX_KEY_DIM = 512
CHUNK_MAX_KEY_DIM = 256   # keys the chunkwise tensor-core kernel takes
SCAN_MAX_TOKENS = 8       # portions up to here run token by token
FINISH_SLICES = 8         # slices of a head a single-token step can finish in one launch (a cluster)
FINISH_CTAS = 400         # ... and does up to this grid: larger ones stream faster as independent CTAs + output kernel


def padded_key_dim(dim: int) -> int:
    if dim > MAX_KEY_DIM:
        raise ValueError(f"matrix-memory keys of {dim} are not supported (at most {MAX_KEY_DIM})")
    return (dim + 15) // 16 * 16


def padded_value_dim(vdim: int) -> int:
    return (vdim + 15) // 16 * 16


@dataclass
class MemoryState:
    """State of one layer run for every request slot; a request's first token finds it as zeros whatever it holds."""
    S: torch.Tensor                     # [slots, heads, dim, vdim]
    n: Optional[torch.Tensor] = None    # [slots, heads, slices, dim]   (retention has no normaliser and maximum)
    m: Optional[torch.Tensor] = None    # [slots, heads, slices]

    @classmethod
    def allocate(cls, slots, heads, dim, vdim, device, gated=True):
        ns = (vdim + SLICE - 1) // SLICE
        z = dict(dtype=torch.float32, device=device)
        S = torch.zeros(slots, heads, dim, vdim, **z)
        return cls(S, torch.zeros(slots, heads, ns, dim, **z), torch.zeros(slots, heads, ns, **z)) if gated else cls(S)

    @staticmethod
    def bytes_per_slot(heads, dim, vdim, gated=True):
        return 4 * heads * (dim * vdim + (((vdim + SLICE - 1) // SLICE) * (dim + 1) if gated else 0))

    def copy_slots(self, src, dst):
        for t in (self.S, self.n, self.m):
            if t is not None:
                t[dst] = t[src]


def _ref(proj, offs, gates, gate_b, cap, q_scale, heads, dim, vdim, rows: StepRows, st: MemoryState):
    q_off, k_off, v_off = offs
    T = proj.shape[0]
    out = torch.zeros(T, heads, vdim)
    g = gates + gate_b
    gi = cap * torch.tanh(g[:, :heads] / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh(g[:, heads:] / cap))
    for t in range(T):
        s, slot = int(rows.row_seq[t]), int(rows.states[rows.row_seq[t]])
        if slot < 0:
            continue
        zero = int(rows.pos[t]) == 0
        S, n, m = (torch.zeros_like(x) if zero else x for x in (st.S[slot], st.n[slot, :, 0], st.m[slot, :, 0]))
        q = proj[t, q_off:q_off + heads * dim].view(heads, dim).float() * q_scale
        k = proj[t, k_off:k_off + heads * dim].view(heads, dim).float()
        v = proj[t, v_off:v_off + heads * vdim].view(heads, vdim).float()
        mn = torch.maximum(gf[t] + m, gi[t])
        keep, put = torch.exp(gf[t] + m - mn), torch.exp(gi[t] - mn)
        S = keep[:, None, None] * S + put[:, None, None] * k[:, :, None] * v[:, None, :]
        n = keep[:, None] * n + put[:, None] * k
        den = torch.maximum((n * q).sum(-1).abs(), torch.exp(-mn)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q) / den[:, None]
        st.S[slot], st.n[slot], st.m[slot] = S, n[:, None].expand_as(st.n[slot]), mn[:, None].expand_as(st.m[slot])
    return out


def _scan(proj, offs, h, gate_w, gates, gate_b, cap, q_scale, heads, dim, vdim, cu, first_pos, slots, st, out=None,
          finish=None, decay=None, turns=None, act=False):
    """Token by token.  ``finish`` = (y, gain, g_off, vdim_true, eps, out_scale): the normed, gated output in place of ``out``.
    ``turns`` / ``act``: queries and keys are rotated, or queries, keys and values pass a silu, as they are read."""
    y, gain, g_off, vdim_true, eps, out_scale = finish if finish is not None else (None, None, 0, vdim, 0.0, 1.0)
    ptrs = (ctypes.c_void_p * 16)(*[t.data_ptr() if t is not None else None for t in
                                    (proj, h, gate_w, gates, gate_b, cu, first_pos, slots, st.S, st.n, st.m, out, y, gain,
                                     decay, turns)])
    dims = (ctypes.c_int * 12)(slots.numel(), *offs, h.shape[1] if h is not None else 0, heads, dim, vdim, g_off, vdim_true,
                               2 * turns.shape[0] if turns is not None else 0, int(act))
    LAUNCHES["matrix_memory"] += 1
    _lib.check(_lib.kernels().gk_matrix_memory_scan(int(proj.dtype == torch.float32), ptrs, proj.stride(0),
                                                    y.stride(0) if y is not None else 0, dims,
                                                    (ctypes.c_float * 4)(cap, q_scale, eps, out_scale), _lib.stream_ptr()),
               "matrix_memory_scan")


def _chunk(proj, offs, gates, gate_b, cap, q_scale, heads, dim, vdim, rows: StepRows, st, out,
           decay=None):
    n = rows.n_portions
    states = rows.states[:n]
    ptrs = (ctypes.c_void_p * 12)(*[t.data_ptr() if t is not None else None for t in
                                    (proj, gates, gate_b, rows.cu, rows.first_pos, states, st.S, st.n, st.m, out,
                                     _lib.err_flag(proj.device), decay)])
    dims = (ctypes.c_int * 8)(n, rows.portion_rows, *offs, heads, dim, vdim)
    LAUNCHES["matrix_memory"] += 1
    _lib.check(_lib.kernels().gk_matrix_memory_chunk(ptrs, proj.stride(0), dims, float(cap), float(q_scale),
                                                     _lib.stream_ptr()), "matrix_memory_chunk")


def _output(o, proj, g_off, gain, vdim_true, eps, y=None, joint=False, out_scale=1.0):
    """Head outputs ``o`` [T, heads, vdim] normed (per head, or ``joint``) and gated: by a sigmoid with a gain, by a silu
    without."""
    T, heads, vdim = o.shape
    if not o.is_cuda:
        if joint:
            n = o.reshape(T, -1)
            n = n * torch.rsqrt(n.pow(2).sum(-1, keepdim=True) / (heads * vdim_true) + eps) * gain * out_scale
            return (n * torch.sigmoid(proj[:, g_off:g_off + heads * vdim].float())).to(proj.dtype)
        n = (o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / vdim_true + eps) * out_scale).reshape(T, -1)
        z = proj[:, g_off:g_off + heads * vdim].float()
        return (n * gain * torch.sigmoid(z) if gain is not None else n * torch.nn.functional.silu(z)).to(proj.dtype)
    LAUNCHES["matrix_memory"] += 1
    if joint:
        dims = (ctypes.c_int * 4)(T, heads * vdim, heads * vdim_true, g_off)
        _lib.check(_lib.kernels().gk_memory_output_joint(
            int(proj.dtype == torch.float32), _lib.ptr(o), _lib.ptr(proj), proj.stride(0), _lib.ptr(gain), _lib.ptr(y),
            y.stride(0), dims, (ctypes.c_float * 2)(eps, out_scale), _lib.stream_ptr()), "memory_output_joint")
        return y
    dims = (ctypes.c_int * 5)(T, heads, vdim, vdim_true, g_off)
    _lib.check(_lib.kernels().gk_memory_output(int(proj.dtype == torch.float32), _lib.ptr(o), _lib.ptr(proj),
                                               proj.stride(0), _lib.ptr(gain), _lib.ptr(y), y.stride(0), dims,
                                               float(eps), float(out_scale), _lib.stream_ptr()), "memory_output")
    return y


def matrix_memory(proj, q_off: int, k_off: int, v_off: int, g_off: int, h, gate_w, gate_b, cap: float, q_scale: float,
                  heads: int, dim: int, vdim: int, vdim_true: int, rows: StepRows, state: MemoryState, gain, eps: float):
    """Runs every row of the step through its request's memory and returns the gated, head-normed output
    [T, heads * vdim].  ``proj``: packed projections; ``h`` [T, width]: the mixer's input, which the 32-bit gate
    projections ``gate_w`` [2 * heads, width] read."""
    T, P = proj.shape[0], rows.portion_rows
    offs = (q_off, k_off, v_off)
    if not proj.is_cuda:
        gates = h.float() @ gate_w.float().t()
        o = _ref(proj, offs, gates, gate_b, cap, q_scale, heads, dim, vdim, rows, state)
        return _output(o, proj, g_off, gain, vdim_true, eps)
    y = torch.empty(T, heads * vdim, dtype=proj.dtype, device=proj.device)
    n = rows.n_portions
    common = (gate_b, cap, q_scale, heads, dim, vdim)
    if P:
        o = torch.empty(P, heads, vdim, dtype=torch.float32, device=proj.device)
        gates = linear_forward(h[:P], gate_w, out_dtype=torch.float32)
        if proj.dtype == torch.bfloat16 and dim <= CHUNK_MAX_KEY_DIM and rows.max_portion > SCAN_MAX_TOKENS:
            _chunk(proj, offs, gates, *common, rows, state, o)
        else:
            _scan(proj, offs, None, None, gates, *common, rows.cu, rows.first_pos, rows.states[:n], state, o)
        _output(o, proj, g_off, gain, vdim_true, eps, y)
    if T > P:
        single = (proj[P:], offs, h[P:], gate_w, None, *common, None, rows.first_pos[n:], rows.states[n:], state)
        slices = (vdim + SLICE - 1) // SLICE
        if slices <= FINISH_SLICES and slices * heads * (T - P) <= FINISH_CTAS:
            _scan(*single, finish=(y[P:], gain, g_off, vdim_true, eps, 1.0))
        else:
            o = torch.empty(T - P, heads, vdim, dtype=torch.float32, device=proj.device)
            _scan(*single, o)
            _output(o, proj[P:], g_off, gain, vdim_true, eps, y[P:])
    return y


def _retention_ref(proj, offs, decay, q_scale, heads, dim, vdim, rows: StepRows, st: MemoryState, turns, act):
    q_off, k_off, v_off = offs
    T = proj.shape[0]
    p = proj.float()
    q, k, v = (p[:, o:o + heads * d].view(T, heads, d) for o, d in ((q_off, dim), (k_off, dim), (v_off, vdim)))
    if turns is not None:
        q, k = (rotate_heads(x, turns, rows.pos) for x in (q, k))
    if act:
        q, k, v = (torch.nn.functional.silu(x) for x in (q, k, v))
    out = torch.zeros(T, heads, vdim)
    for t in range(T):
        slot = int(rows.states[rows.row_seq[t]])
        if slot < 0:
            continue
        S = torch.zeros_like(st.S[slot]) if int(rows.pos[t]) == 0 else st.S[slot]
        st.S[slot] = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", st.S[slot], q[t]) * q_scale
    return out


def retention(proj, q_off: int, k_off: int, v_off: int, g_off: int, decay, q_scale: float, heads: int, dim: int, vdim: int,
              vdim_true: int, rows: StepRows, state: MemoryState, eps: float, y, turns=None, act: bool = False, gain=None,
              out_scale: float = 1.0):
    """Retention over the rows of a step: ``S <- decay_h S + k v^T``, head output ``S^T q * q_scale`` divided by its root
    mean square (over ``vdim_true`` columns) and multiplied by ``silu(g)``; with ``gain`` [heads * vdim], all heads' outputs
    divided by their common root mean square and multiplied by ``gain * sigmoid(g)``.  Times ``out_scale``, written to ``y``
    [T, heads * vdim] (any row stride).  ``decay``: [heads] 32-bit.  Queries and keys are rotated with ``turns`` (neighbours
    paired), or queries, keys and values pass a silu with ``act``; both may happen in place."""
    T, P, n = proj.shape[0], rows.portion_rows, rows.n_portions
    offs = (q_off, k_off, v_off)
    joint = gain is not None
    if not proj.is_cuda:
        o = _retention_ref(proj, offs, decay, q_scale, heads, dim, vdim, rows, state, turns, act)
        y.copy_(_output(o, proj, g_off, gain, vdim_true, eps, joint=joint, out_scale=out_scale))
        return y
    common = (None, None, 0.0, q_scale, heads, dim, vdim)
    f32 = dict(dtype=torch.float32, device=proj.device)
    if P:
        o = torch.empty(P, heads, vdim, **f32)
        if turns is not None:
            head_prep(proj, rows, 0, P, q_off, heads, k_off, heads, dim, turns=turns)
        if act:
            sizes = (heads * dim, heads * dim, heads * vdim)
            if offs == (q_off, q_off + sizes[0], q_off + sizes[0] + sizes[1]):
                silu_columns(proj[:P], q_off, sum(sizes))
            else:
                for at, size in zip(offs, sizes):
                    silu_columns(proj[:P], at, size)
        if proj.dtype == torch.bfloat16 and dim <= CHUNK_MAX_KEY_DIM and rows.max_portion > SCAN_MAX_TOKENS:
            _chunk(proj, offs, *common, rows, state, o, decay)
        else:
            _scan(proj, offs, None, None, *common, rows.cu, rows.first_pos, rows.states[:n], state, o, decay=decay)
        _output(o, proj, g_off, gain, vdim_true, eps, y[:P], joint, out_scale)
    if T > P:
        single = (proj[P:], offs, None, None, *common, None, rows.first_pos[n:], rows.states[n:], state)
        slices = (vdim + SLICE - 1) // SLICE
        if not joint and slices <= FINISH_SLICES and slices * heads * (T - P) <= FINISH_CTAS:
            _scan(*single, finish=(y[P:], None, g_off, vdim_true, eps, out_scale), decay=decay, turns=turns, act=act)
        else:
            o = torch.empty(T - P, heads, vdim, **f32)
            _scan(*single, o, decay=decay, turns=turns, act=act)
            _output(o, proj[P:], g_off, gain, vdim_true, eps, y[P:], joint, out_scale)
    return y

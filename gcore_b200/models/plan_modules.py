"""Parts that layer-plan decoders share: mixers and feed-forwards that read their columns of a packed input projection and
write their columns of the matrix an output projection reads.  ``load`` takes a part's tensors from a checkpoint into its
rows of the one projection and its columns of the other.

Every block of columns is a multiple of 8 wide and heads are padded with zero rows to the sizes the kernels store; zero
padding changes no score, state or output, and means are taken over the true sizes."""
from __future__ import annotations

import math

import torch
import torch.nn as nn

from ..ops import diff_attention as da, latent_attention as la, matrix_memory as mm, moe, scored_attention as sa
from .layer_plan import (DenseSpec, DifferentialAttentionSpec, ExpertsSpec, LatentAttentionSpec, RetentionSpec,
                         ScoredAttentionSpec)
from .plan_decoder import _buf, _up, put, put_heads


def blocks(*sizes):
    """Offsets of consecutive blocks and their total."""
    at, n = [], 0
    for s in sizes:
        at.append(n)
        n += s
    return at, n


class LatentAttentionMixer(nn.Module):
    def __init__(self, spec: LatentAttentionSpec, width: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.width = spec, width
        rank, rot = la.cached_row(spec.kv_rank, spec.rot_dim)
        dim, vdim = _up(spec.dim, 8), _up(spec.vdim, 8)
        per_head = vdim if spec.gate == "element" else 1            # gate columns
        (q, down, gate), self.columns = blocks(spec.heads * (dim + rot), rank + rot, _up(spec.heads * per_head, 8))
        self.layout = la.LatentLayout(q=q, down=down, gate=gate, heads=spec.heads, dim=dim, vdim=vdim, rank=spec.kv_rank,
                                      row_rank=rank, rot=spec.rot_dim, row_rot=rot, scale=spec.scale,
                                      magnitude=spec.rot.magnitude(), eps=eps, window=spec.window, gate_cols=per_head)
        self.out_columns = spec.heads * vdim
        self.gain = _buf(torch.zeros(spec.kv_rank, dtype=torch.float32, device=device))
        self.turns = _buf(la.rotation_turns(spec.rot.frequencies()).to(device))
        self.up_kv = _buf(torch.zeros(spec.heads * (dim + vdim), rank, dtype=dtype, device=device))
        self.sinks = _buf(torch.zeros(spec.heads, dtype=torch.float32, device=device)) if spec.sink else None

    def cache_shape(self):
        return 1, self.layout.row

    def new_state(self, slots, device):
        return None

    def state_bytes(self):
        return 0

    def load(self, take, p: str, rows, out, bias=None):
        s, ly, W = self.spec, self.layout, self.width
        H, d, r, C = s.heads, s.dim, s.rot_dim, s.kv_rank
        q = take(p + "q", H * (d + r), W).view(H, d + r, W)
        dst = rows[ly.q:ly.q + H * (ly.dim + ly.row_rot)].view(H, ly.dim + ly.row_rot, -1)
        put(dst, q[:, :d])
        put(dst[:, ly.dim:], q[:, d:])
        down = take(p + "dkv", C + r, W)
        put(rows[ly.down:], down[:C])
        put(rows[ly.down + ly.row_rank:], down[C:])
        if s.gate == "element":
            put_heads(rows[ly.gate:ly.gate + H * ly.vdim], take(p + "g", H * s.vdim, W), H, s.vdim, ly.vdim)
        else:
            put(rows[ly.gate:], take(p + "g", H, W))
        if self.sinks is not None:
            put(self.sinks, take(p + "sink", H).float())
        put(self.gain, take(p + "dkv.norm", C).float())
        put_heads(self.up_kv[:H * ly.dim], take(p + "uk", H * d, C), H, d, ly.dim)
        put_heads(self.up_kv[H * ly.dim:], take(p + "uv", H * s.vdim, C), H, s.vdim, ly.vdim)
        put(out.view(out.shape[0], H, ly.vdim), take(p + "o", W, H * s.vdim).view(W, H, s.vdim))

    def forward(self, proj, rows, cache, state, out):
        la.latent_attention(proj, self.layout, self.gain, self.turns, self.up_kv, rows, cache, out, self.sinks)


class DifferentialAttentionMixer(nn.Module):
    """Its projections have biases (``biased``): that of the input projection is loaded with the rows, that of the output
    projection by the layer."""
    biased = True

    def __init__(self, spec: DifferentialAttentionSpec, width: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.width = spec, width
        H, G, dim, vdim = spec.heads, spec.kv_heads, _up(spec.dim, 8), _up(spec.vdim, 8)
        (q, k, v, gate), self.columns = blocks(H * 2 * dim, G * 2 * dim, G * vdim, _up(H, 8))
        self.layout = da.DiffLayout(q=q, k=k, v=v, gate=gate, heads=H, kv_heads=G, dim=dim, vdim=vdim, true_vdim=spec.vdim,
                                    rot=spec.rot.dims, magnitude=spec.rot.magnitude(), scale=spec.scale,
                                    out_scale=1.0 - spec.diff, eps=eps)
        self.out_columns = H * vdim
        self.turns = _buf(la.rotation_turns(spec.rot.frequencies()).to(device))
        self.lam = _buf(torch.zeros(1, dtype=torch.float32, device=device))      # weight of the second map

    def cache_shape(self):
        return (self.layout.row,)

    def new_state(self, slots, device):
        return None

    def state_bytes(self):
        return 0

    def load(self, take, p: str, rows, out, bias):
        s, ly, W = self.spec, self.layout, self.width
        for at, nm, n, dim, pad in ((ly.q, "q", 2 * s.heads, s.dim, ly.dim), (ly.k, "k", 2 * s.kv_heads, s.dim, ly.dim),
                                    (ly.v, "v", s.kv_heads, s.vdim, ly.vdim)):
            put_heads(rows[at:at + n * pad], take(p + nm, n * dim, W), n, dim, pad)
            put_heads(bias[at:at + n * pad], take(p + nm + ".b", n * dim).float(), n, dim, pad)
        put(rows[ly.gate:], take(p + "g", s.heads, W))
        lq1, lk1, lq2, lk2 = (take(p + nm, s.dim).double() for nm in ("lq1", "lk1", "lq2", "lk2"))
        self.lam.fill_(math.exp(float(lq1 @ lk1)) - math.exp(float(lq2 @ lk2)) + s.diff)
        put(out.view(out.shape[0], s.heads, ly.vdim), take(p + "o", W, s.heads * s.vdim).view(W, s.heads, s.vdim))

    def forward(self, proj, rows, cache, state, out):
        da.differential_attention(proj, self.layout, self.turns, self.lam, rows, cache, out)


def _head_order(rot, dim: int):
    """Dimensions of a head in the order the kernels rotate (neighbours paired), or None if that is their own order."""
    return rot.neighbours(dim) if rot is not None and rot.halves else None


def _take_heads(take, name: str, heads: int, dim: int, width: int, order=None):
    t = take(name, heads * dim, width)
    return t if order is None else t.view(heads, dim, width)[:, order].reshape(heads * dim, width)


class ScoredAttentionMixer(nn.Module):
    def __init__(self, spec: ScoredAttentionSpec, width: int, eps: float, dtype, device, out_scale: float = 1.0):
        super().__init__()
        self.spec, self.width, self.out_scale = spec, width, out_scale
        H, G, dim, vdim = spec.heads, spec.kv_heads, _up(spec.dim, 8), _up(spec.vdim, 8)
        (q, k, v), self.columns = blocks(H * dim, G * dim, G * vdim)
        self.layout = sa.ScoredLayout(q=q, k=k, v=v, heads=H, kv_heads=G, dim=dim, true_dim=spec.dim, vdim=vdim, scale=spec.scale,
                                      eps=eps, unit=spec.unit, sigmoid=spec.weights == "sigmoid", window=spec.window,
                                      keep=spec.keep if spec.window else 0)
        self.out_columns = H * vdim
        f32 = dict(dtype=torch.float32, device=device)
        self.turns = _buf(la.rotation_turns(spec.rot.frequencies()).to(device)) if spec.rot is not None else None
        self.r1, self.r2 = (_buf(torch.zeros(H, **f32)) if spec.distance else None for _ in range(2))
        self.head_bias = _buf(torch.zeros(H, **f32)) if spec.head_bias else None

    def cache_shape(self):
        return (self.layout.row,)

    def new_state(self, slots, device):
        return None

    def state_bytes(self):
        return 0

    def load(self, take, p: str, rows, out):
        s, ly, W = self.spec, self.layout, self.width
        order = _head_order(s.rot, s.dim)
        for at, nm, n, dim, pad, o in ((ly.q, "q", s.heads, s.dim, ly.dim, order), (ly.k, "k", s.kv_heads, s.dim, ly.dim, order),
                                       (ly.v, "v", s.kv_heads, s.vdim, ly.vdim, None)):
            put_heads(rows[at:at + n * pad], _take_heads(take, p + nm, n, dim, W, o), n, dim, pad)
        for nm, dst in (("r1", self.r1), ("r2", self.r2), ("pb", self.head_bias)):
            if dst is not None:
                put(dst, take(p + nm, s.heads).float())
        put(out.view(out.shape[0], s.heads, ly.vdim), take(p + "o", W, s.heads * s.vdim).view(W, s.heads, s.vdim))

    def forward(self, proj, rows, cache, state, out):
        sa.scored_attention(proj, self.layout, rows, cache, out, self.turns, (self.r1, self.r2) if self.spec.distance else None,
                            self.head_bias, self.out_scale)


class RetentionMixer(nn.Module):
    def __init__(self, spec: RetentionSpec, width: int, eps: float, dtype, device, out_scale: float = 1.0):
        super().__init__()
        self.spec, self.width, self.eps, self.out_scale = spec, width, eps, out_scale
        self.dim, self.vdim = mm.padded_key_dim(spec.dim), mm.padded_value_dim(spec.vdim)
        H = spec.heads
        self.at, self.columns = blocks(H * self.dim, H * self.dim, H * self.vdim, H * self.vdim)
        self.out_columns = H * self.vdim
        f32 = dict(dtype=torch.float32, device=device)
        self.decay = _buf(torch.tensor(spec.decay, **f32))
        self.turns = _buf(la.rotation_turns(spec.rot.frequencies()).to(device)) if spec.rot is not None else None
        self.gain = _buf(torch.zeros(H * self.vdim, **f32)) if spec.norm == "joint" else None

    def cache_shape(self):
        return None

    def new_state(self, slots, device):
        return mm.MemoryState.allocate(slots, self.spec.heads, self.dim, self.vdim, device, gated=False)

    def state_bytes(self):
        return mm.MemoryState.bytes_per_slot(self.spec.heads, self.dim, self.vdim, gated=False)

    def load(self, take, p: str, rows, out):
        s, W, H = self.spec, self.width, self.spec.heads
        order = _head_order(s.rot, s.dim)
        for at, nm, dim, pad, o in zip(self.at, "qkvg", (s.dim, s.dim, s.vdim, s.vdim),
                                       (self.dim, self.dim, self.vdim, self.vdim), (order, order, None, None)):
            put_heads(rows[at:at + H * pad], _take_heads(take, p + nm, H, dim, W, o), H, dim, pad)
        if self.gain is not None:
            put_heads(self.gain, take(p + "norm", H * s.vdim).float(), H, s.vdim, self.vdim)
        put(out.view(out.shape[0], H, self.vdim), take(p + "o", W, H * s.vdim).view(W, H, s.vdim))

    def forward(self, proj, rows, cache, state, out):
        s = self.spec
        mm.retention(proj, *self.at, self.decay, s.product_scale(), s.heads, self.dim, self.vdim, s.vdim, rows, state, self.eps,
                     out, self.turns, s.act == "silu", self.gain, self.out_scale)


class DenseFeedForward(nn.Module):
    def __init__(self, spec: DenseSpec, width: int, width_pad: int, dtype, device):
        super().__init__()
        self.spec, self.width, self.ff = spec, width, _up(spec.ff, 8)
        self.gated = spec.act == "silu_gate"
        self.columns, self.out_columns = (2 if self.gated else 1) * self.ff, self.ff

    def load(self, take, p: str, rows, out):
        f, W = self.spec.ff, self.width
        if self.gated:
            put(rows, take(p + "gate", f, W))
        put(rows[self.columns - self.ff:], take(p + "up", f, W))
        put(out, take(p + "down", W, f))

    def forward(self, h, proj, out, counts):
        if self.gated:
            moe.activate(moe.SILU_GATE, proj, self.ff, self.ff, out)
        else:
            moe.activate(moe.RELU2, proj, self.ff, 0, out)
        return None


class ExpertFeedForward(nn.Module):
    """The shared expert is part of the projections around it; routed experts run on the grouped GEMM."""

    def __init__(self, spec: ExpertsSpec, width: int, width_pad: int, dtype, device):
        super().__init__()
        if spec.experts > moe.MAX_EXPERTS or spec.top > moe.MAX_TOP:
            raise ValueError(f"at most {moe.MAX_EXPERTS} experts and {moe.MAX_TOP} choices are supported")
        if spec.groups > moe.MAX_GROUPS:
            raise ValueError(f"at most {moe.MAX_GROUPS} expert groups are supported")
        self.spec, self.width = spec, width
        self.ff, self.shared = _up(spec.ff, 8), _up(spec.shared_ff, 8)
        self.act = moe.SILU_GATE if spec.act == "silu_gate" else moe.RELU2
        mats = 2 if spec.act == "silu_gate" else 1                  # input matrices of an expert: [gate |] up
        self.columns, self.out_columns = mats * self.shared, self.shared
        self.how = dict(sigmoid=spec.score == "sigmoid", norm=spec.normalize, scale=spec.scale, groups=spec.groups,
                        keep=spec.keep)
        self.gate_row = 1 if self.shared and spec.shared_gate else 0        # the shared expert's gate behind the router
        act = dict(dtype=dtype, device=device)
        E = spec.experts
        self.router = _buf(torch.zeros(E + self.gate_row, width_pad, **act))
        self.correction = _buf(torch.zeros(E, dtype=torch.float32, device=device))
        self.up = _buf(torch.zeros(E, mats * self.ff, width_pad, **act))
        self.down = _buf(torch.zeros(E, width_pad, self.ff, **act))

    def load(self, take, p: str, rows, out):
        s, W = self.spec, self.width
        put(self.router, take(p + "router", s.experts, W))
        put(self.correction, take(p + "correction", s.experts).float())
        names = ("gate", "up") if s.act == "silu_gate" else ("up",)
        for e in range(s.experts):
            for k, nm in enumerate(names):
                put(self.up[e, k * self.ff:], take(f"{p}e{e}.{nm}", s.ff, W))
            put(self.down[e], take(f"{p}e{e}.down", W, s.ff))
        if self.shared:
            for k, nm in enumerate(names):
                put(rows[k * self.shared:], take(p + "shared." + nm, s.shared_ff, W))
            put(out, take(p + "shared.down", W, s.shared_ff))
        if self.gate_row:
            put(self.router[s.experts:], take(p + "shared.sg", 1, W))

    def forward(self, h, proj, out, counts):
        s = self.spec
        logits, choice = moe.route_tokens(h, self.router, s.experts, s.top, self.correction, counts, **self.how)
        if self.shared:
            moe.activate(self.act, proj, self.shared, self.shared if self.act == moe.SILU_GATE else 0, out,
                         row_logit=logits[:, s.experts] if self.gate_row else None)
        return moe.routed_experts(h, choice, self.up, self.down, counts, self.act)

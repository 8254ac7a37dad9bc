"""Serving modules of layer-plan decoders whose sublayers read their normed input through a short causal convolution
(Rezulorn): pre-norm layers with one mixer, or a weighted sum of two, and a feed-forward.

A sublayer is an input projection, the part on its columns, and an output projection; what lies between two sublayers - the
residual, its norm and the convolution - is one launch (``ops/conv_norm.py``).  Mixers side by side read the same input and are
summed, so their input matrices are one, and ``[output of one | output of the other]`` times ``[W_o | W_o']`` is the sum; the
scales are applied to the outputs, in 32-bit.  A request's state in a layer is the recurrent mixer's and the last inputs of both
convolutions."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from ..ops import conv_norm as cn
from ..ops.gemm import linear_forward
from ..ops.matrix_memory import MemoryState
from .config import ModelConfig
from .layer_plan import ConvLayerSpec, RetentionSpec
from .plan_decoder import CheckpointTensors, PlanDecoder, _buf, put
from .plan_modules import DenseFeedForward, RetentionMixer, ScoredAttentionMixer


@dataclass
class ConvLayerState:
    """State of one layer run for every request slot."""
    rings: list                              # per sublayer: [slots, taps - 1, width], last inputs of its convolution
    memory: Optional[MemoryState] = None     # recurrent mixer

    def copy_slots(self, src, dst):
        for t in self.rings:
            t[dst] = t[src]
        if self.memory is not None:
            self.memory.copy_slots(src, dst)


class ConvSublayer(nn.Module):
    """Parts that read the same input and are summed, their projections, norm and convolution."""

    def __init__(self, parts, width: int, width_pad: int, taps: int, dtype, device):
        super().__init__()
        self.parts, self.width, self.n_taps = nn.ModuleList(parts), width, taps
        act, f32 = dict(dtype=dtype, device=device), dict(dtype=torch.float32, device=device)
        self.in_proj = _buf(torch.zeros(sum(p.columns for p in parts), width_pad, **act))
        self.out_proj = _buf(torch.zeros(width_pad, sum(p.out_columns for p in parts), **act))
        self.gain = _buf(torch.zeros(width_pad, **f32))
        # [taps, width]; the present's tap holds 1 + w, since a sublayer reads its input plus the convolution
        self.taps = _buf(torch.zeros(cn.stored_taps(taps), width_pad, **f32))

    def load(self, take, p: str, q: int, names):
        put(self.gain, take(f"{p}norm{q}", self.width).float())
        put(self.taps[self.taps.shape[0] - self.n_taps:], take(f"{p}canon{q}", self.width, self.n_taps).float().t())
        self.taps[-1, :self.width] += 1
        n = k = 0
        for part, name in zip(self.parts, names):
            part.load(take, p + name, self.in_proj[n:n + part.columns], self.out_proj[:, k:k + part.out_columns])
            n, k = n + part.columns, k + part.out_columns

    def project_in(self, h):
        """Packed columns of the parts, and an empty matrix for their outputs."""
        return linear_forward(h, self.in_proj), torch.empty(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)

    def columns(self, proj, out):
        """Every part with its columns of both matrices."""
        n = k = 0
        for part in self.parts:
            yield part, proj[:, n:n + part.columns], out[:, k:k + part.out_columns]
            n, k = n + part.columns, k + part.out_columns


class ConvLayer(nn.Module):
    def __init__(self, spec: ConvLayerSpec, taps: int, width: int, width_pad: int, eps: float, dtype, device):
        super().__init__()
        # checkpoint names of the mixers: alone, or side by side
        self.names = ("mix.",) if len(spec.mixers) == 1 else ("mix.left.", "mix.right.")
        if len(spec.mixers) > 2 or sum(isinstance(m, RetentionSpec) for m in spec.mixers) > 1 or \
                sum(not isinstance(m, RetentionSpec) for m in spec.mixers) > 1:
            raise ValueError("a layer runs at most one attention and one recurrent mixer")
        parts = [(RetentionMixer if isinstance(m, RetentionSpec) else ScoredAttentionMixer)(m, width, eps, dtype, device, scale)
                 for m, scale in zip(spec.mixers, spec.scales)]
        self.mixer = ConvSublayer(parts, width, width_pad, taps, dtype, device)
        self.ffn = None
        if spec.ffn is not None:
            self.ffn = ConvSublayer([DenseFeedForward(spec.ffn, width, width_pad, dtype, device)], width, width_pad, taps, dtype,
                                    device)

    def _part(self, cls):
        return next((p for p in self.mixer.parts if isinstance(p, cls)), None)

    def sublayers(self):
        return [s for s in (self.mixer, self.ffn) if s is not None]

    def cache_shape(self):
        attention = self._part(ScoredAttentionMixer)
        return attention.cache_shape() if attention is not None else None

    def new_state(self, slots, device):
        memory = self._part(RetentionMixer)
        rings = [torch.zeros(slots, s.taps.shape[0] - 1, s.taps.shape[1], dtype=torch.float32, device=device)
                 for s in self.sublayers()]
        return ConvLayerState(rings, memory.new_state(slots, device) if memory is not None else None)

    def state_bytes(self):
        memory = self._part(RetentionMixer)
        rings = sum(4 * (s.taps.shape[0] - 1) * s.taps.shape[1] for s in self.sublayers())
        return rings + (memory.state_bytes() if memory is not None else 0)

    def load(self, take, p: str):
        self.mixer.load(take, p, 1, self.names)
        if self.ffn is not None:
            self.ffn.load(take, p, 2, ("mlp.",))
        else:       # without the sublayer its norm and convolution mean nothing
            take.drop(p + "norm2", p + "canon2")

    def mix_tokens(self, h, rows, cache, state):
        proj, act = self.mixer.project_in(h)
        for part, columns, out in self.mixer.columns(proj, act):
            part(columns, rows, cache, state.memory, out)
        return linear_forward(act, self.mixer.out_proj)

    def feed_forward(self, h):
        proj, act = self.ffn.project_in(h)
        self.ffn.parts[0](h, proj, act, None)
        return linear_forward(act, self.ffn.out_proj)


class ConvDecoder(PlanDecoder):
    def __init__(self, cfg: ModelConfig, device=None):
        if cfg.hidden_size > cn.MAX_WIDTH:
            raise ValueError(f"widths up to {cn.MAX_WIDTH} are supported, not {cfg.hidden_size}")
        super().__init__(cfg, device)
        self.norm = cn.NormSpec(self.width, cfg.rms_norm_eps)
        self.head = _buf(torch.zeros(cfg.vocab_size, self.width_pad, dtype=self.dtype, device=device))

    @property
    def output_weight(self):
        return self.head

    def make_layer(self, index, spec, device):
        return ConvLayer(spec, self.cfg.layer_plan.taps, self.width, self.width_pad, self.cfg.rms_norm_eps, self.dtype, device)

    @torch.no_grad()
    def load_tensors(self, tensors):
        """Fills the module from a Rezulorn checkpoint's tensors (``embed``, ``l<i>.norm1``, ``l<i>.canon1``, ``l<i>.mix.q`` or
        ``l<i>.mix.left.q`` ..., ``l<i>.mlp.up`` ..., ``final.norm``, ``head``); every tensor must be there with its configured
        shape and none may be left over.  The factor of the logits becomes part of the final gain."""
        take = CheckpointTensors(tensors)
        put(self.embed, take("embed", self.cfg.vocab_size, self.width))
        put(self.head, take("head", self.cfg.vocab_size, self.width))
        put(self.final_gain, take("final.norm", self.width).float() * self.cfg.layer_plan.logit_scale)
        for i, layer in enumerate(self.layers):
            layer.load(take, f"l{i}.")
        take.done()
        return self

    @torch.no_grad()
    def randomize(self, seed: int = 0):
        """Random weights of the right scale (benchmarks); padding is not kept apart."""
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("turns", "decay"):
                continue
            if leaf == "taps":
                p.normal_(0.0, 0.2, generator=g)
                p[-1] += 1
            elif leaf == "head_bias":
                p.fill_(-4.0)
            elif p.dim() == 1:
                p.fill_(0.5 if leaf in ("r1", "r2") else 1.0)
            else:
                p.normal_(0.0, 1.0 if name == "embed" else 1.0 / math.sqrt(p.shape[-1]), generator=g)
        return self

    def final_rows(self, x, rows=None):
        return cn.conv_norm_rows(x, self.final_gain, self.norm, self.embed.dtype, rows)

    def forward(self, rows, caches, states, final=True, record=None):
        runs, mult, spec = self.cfg.layer_plan.runs, self.cfg.layer_plan.residual_mult, self.norm
        subs = [(s, states[r.index].rings[k]) for r in runs for k, s in enumerate(self.layers[r.layer].sublayers())]
        first, ring = subs[0]
        x, h = cn.conv_embed_rows(rows, self.embed, first.gain, first.taps, ring, spec)
        at = 0

        def join(y):
            """Behind a sublayer: the residual, and the input of the next one (or the final norm at the end)."""
            nonlocal x, h, at
            at += 1
            if at < len(subs):
                sub, ring = subs[at]
                x, h = cn.conv_add_sublayer(x, y, mult, spec, sub.gain, rows, sub.taps, ring)
            else:
                x, h = cn.conv_add_sublayer(x, y, mult, spec, self.final_gain if final else None, keep=not final or record is not None)

        for r in runs:
            layer = self.layers[r.layer]
            join(layer.mix_tokens(h, rows, caches[r.index], states[r.index]))
            if layer.ffn is not None:
                join(layer.feed_forward(h))
            if record is not None:
                record.append(x.clone())
        return h if final else x

"""Serving modules of layer-plan decoders whose layers run one mixer and one feed-forward side by side on the same normed
input and hand on a weighted average over depth (Kedesun).

Because both sublayers read the same input and are summed, a layer has two projections only: one into
``[mixer columns | feed-forward columns]`` and one out of ``[mixer output | feed-forward activation]``, whose product is the
sum of the two.  Routed experts are added to it, still in expert order, by the residual step."""
from __future__ import annotations

import math

import torch
import torch.nn as nn

from ..ops import depth, sandwich
from ..ops.gemm import linear_forward
from .config import ModelConfig
from .layer_plan import ExpertsSpec, LatentAttentionSpec, ParallelLayerSpec
from .plan_decoder import CheckpointTensors, PlanDecoder, _buf, put
from .plan_modules import DenseFeedForward, ExpertFeedForward, LatentAttentionMixer, RetentionMixer


class ParallelLayer(nn.Module):
    """One layer's weights and its forward over the rows of a step."""

    def __init__(self, index: int, spec: ParallelLayerSpec, width: int, width_pad: int, eps: float, dtype, device):
        super().__init__()
        self.index, self.width = index, width
        mixer = LatentAttentionMixer if isinstance(spec.mixer, LatentAttentionSpec) else RetentionMixer
        self.mixer = mixer(spec.mixer, width, eps, dtype, device)
        self.ffn = None
        if spec.ffn is not None:
            ffn = ExpertFeedForward if isinstance(spec.ffn, ExpertsSpec) else DenseFeedForward
            self.ffn = ffn(spec.ffn, width, width_pad, dtype, device)
        self.experts = spec.ffn.experts if isinstance(spec.ffn, ExpertsSpec) else 0
        n, k = self.mixer.columns, self.mixer.out_columns
        if self.ffn is not None:
            n, k = n + self.ffn.columns, k + self.ffn.out_columns
        self.in_proj = _buf(torch.zeros(n, width_pad, dtype=dtype, device=device))
        self.out_proj = _buf(torch.zeros(width_pad, k, dtype=dtype, device=device))
        self.pre = _buf(torch.zeros(width_pad, dtype=torch.float32, device=device))
        self.avg = _buf(torch.zeros(index + 2, dtype=torch.float32, device=device))

    def cache_shape(self):
        return self.mixer.cache_shape()

    def new_state(self, slots, device):
        return self.mixer.new_state(slots, device)

    def state_bytes(self):
        return self.mixer.state_bytes()

    def load(self, take, p: str):
        put(self.pre, take(p + "norm1", self.width).float())
        put(self.avg, take(p + "dwa", self.index + 2).float())
        n, k = self.mixer.columns, self.mixer.out_columns
        self.mixer.load(take, p + "mix.", self.in_proj[:n], self.out_proj[:, :k])
        if self.ffn is not None:
            self.ffn.load(take, p + "mlp.", self.in_proj[n:], self.out_proj[:, k:])

    def forward(self, h, rows, cache, state, counts):
        """``h``: normed input.  Returns the layer's summed update and the routed experts' part of it (or None)."""
        proj = linear_forward(h, self.in_proj)
        act = torch.empty(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)
        n, k = self.mixer.columns, self.mixer.out_columns
        self.mixer(proj, rows, cache, state, act[:, :k])
        routed = self.ffn(h, proj[:, n:], act[:, k:], counts) if self.ffn is not None else None
        return linear_forward(act, self.out_proj), routed


class ParallelDecoder(PlanDecoder):
    """Output matrix = embedding table."""

    def __init__(self, cfg: ModelConfig, device=None):
        if cfg.layer_plan.loop_times:
            raise ValueError("a weighted average over depth and looped layers do not go together")
        super().__init__(cfg, device)

    @property
    def output_weight(self):
        return self.embed

    def make_layer(self, index, spec, device):
        return ParallelLayer(index, spec, self.width, self.width_pad, self.cfg.rms_norm_eps, self.dtype, device)

    @torch.no_grad()
    def load_tensors(self, tensors):
        """Fills the module from a Kedesun checkpoint's tensors (``embed``, ``l<i>.norm1``, ``l<i>.mix.q`` ...,
        ``l<i>.mlp.e<j>.up`` ..., ``l<i>.dwa``, ``final.norm``); every tensor must be there with its configured shape and
        none may be left over."""
        take = CheckpointTensors(tensors)
        put(self.embed, take("embed", self.cfg.vocab_size, self.width))
        put(self.final_gain, take("final.norm", self.width).float())
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
            if leaf == "avg":
                p.fill_(0.3 / p.numel())
                p[-1] = 0.7
            elif leaf == "correction":
                p.normal_(0.0, 0.01, generator=g)
            elif p.dim() == 1:
                p.fill_(1.0)
            else:
                p.normal_(0.0, 1.0 if name == "embed" else 1.0 / math.sqrt(p.shape[-1]), generator=g)
        return self

    def forward(self, rows, caches, states, final=True, record=None):
        L, eps, W, T = len(self.layers), self.cfg.rms_norm_eps, self.width, rows.tokens.numel()
        f32 = dict(dtype=torch.float32, device=self.embed.device)
        history = torch.empty(L, T, self.width_pad, **f32)
        x = torch.empty(T, self.width_pad, **f32)
        experts = [ly.experts for ly in self.layers]
        counts = None
        if any(experts):     # cleared once per step for all layers
            counts = torch.zeros(L, max(experts), dtype=torch.int32, device=self.embed.device)
        _, _, h = sandwich.embed_rows(rows.tokens, rows.pos, self.embed, None, self.layers[0].pre, W, eps, x=history[0])
        for i, layer in enumerate(self.layers):
            y, routed = layer(h, rows, caches[i], states[i], counts[i, :experts[i]] if experts[i] else None)
            last = i + 1 == L
            gain = (self.final_gain if final else None) if last else self.layers[i + 1].pre
            h = depth.add_layer(history, i + 1, x if i else history[0], y, layer.avg, W, eps, x, gain, routed, keep=not last)
            if record is not None:
                record.append(x.clone())
        return h if final else x

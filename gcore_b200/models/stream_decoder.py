"""Serving modules of layer-plan decoders with hyper-connections (Lobutar): several 32-bit residual streams, of which every
sublayer reads one weighted sum and writes to all, mixing them on the way.

A sublayer is an input projection, the mixer or feed-forward on its columns, and an output projection; what lies between two
sublayers - the write, the mixture, the next read and its norm - is one launch (``ops/streams.py``).  Routed experts are added
there, still in expert order."""
from __future__ import annotations

import math

import torch
import torch.nn as nn

from ..ops import streams as hc
from ..ops.gemm import linear_forward
from .config import ModelConfig
from .layer_plan import DifferentialAttentionSpec, ExpertsSpec, StreamLayerSpec
from .plan_decoder import CheckpointTensors, PlanDecoder, _buf, put
from .plan_modules import DenseFeedForward, DifferentialAttentionMixer, ExpertFeedForward, LatentAttentionMixer


class Sublayer(nn.Module):
    """A part (mixer or feed-forward), its projections (``None`` where it has no columns), norm and connections."""

    def __init__(self, part: nn.Module, streams: int, width: int, width_pad: int, dtype, device):
        super().__init__()
        self.part, self.width, self.streams = part, width, streams
        f32, act = dict(dtype=torch.float32, device=device), dict(dtype=dtype, device=device)
        self.in_proj = _buf(torch.zeros(part.columns, width_pad, **act)) if part.columns else None
        self.out_proj = _buf(torch.zeros(width_pad, part.out_columns, **act)) if part.out_columns else None
        biased = getattr(part, "biased", False)
        self.in_bias = _buf(torch.zeros(part.columns, **f32)) if biased else None
        self.out_bias = _buf(torch.zeros(width_pad, **f32)) if biased else None
        self.gain = _buf(torch.zeros(width_pad, **f32))
        self.read = _buf(torch.zeros(streams, **f32))
        self.write = _buf(torch.zeros(streams, **f32))
        self.mix = _buf(torch.zeros(streams, streams, **f32))        # [from, to]

    def load(self, take, p: str, q: int, part: str):
        S, W = self.streams, self.width
        put(self.gain, take(f"{p}norm{q}", W).float())
        for dst, nm, shape in ((self.read, "in", (S,)), (self.write, "out", (S,)), (self.mix, "mix", (S, S))):
            put(dst, take(f"{p}hc{q}.{nm}", *shape).float())
        if self.in_bias is not None:
            self.part.load(take, p + part, self.in_proj, self.out_proj, self.in_bias)
            put(self.out_bias, take(p + part + "o.b", W).float())
        else:
            self.part.load(take, p + part, self.in_proj, self.out_proj)

    def project_in(self, h):
        """Packed columns of the part, and an empty matrix for its output."""
        if self.in_proj is None:
            return None, None
        return linear_forward(h, self.in_proj, self.in_bias), \
            torch.empty(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)

    def project_out(self, act):
        return linear_forward(act, self.out_proj, self.out_bias) if act is not None else None


class StreamLayer(nn.Module):
    def __init__(self, spec: StreamLayerSpec, streams: int, width: int, width_pad: int, eps: float, dtype, device):
        super().__init__()
        mixer = DifferentialAttentionMixer if isinstance(spec.mixer, DifferentialAttentionSpec) else LatentAttentionMixer
        self.mixer = Sublayer(mixer(spec.mixer, width, eps, dtype, device), streams, width, width_pad, dtype, device)
        self.ffn = None
        if spec.ffn is not None:
            ffn = ExpertFeedForward if isinstance(spec.ffn, ExpertsSpec) else DenseFeedForward
            self.ffn = Sublayer(ffn(spec.ffn, width, width_pad, dtype, device), streams, width, width_pad, dtype, device)
        self.experts = spec.ffn.experts if isinstance(spec.ffn, ExpertsSpec) else 0

    def cache_shape(self):
        return self.mixer.part.cache_shape()

    def new_state(self, slots, device):
        return self.mixer.part.new_state(slots, device)

    def state_bytes(self):
        return self.mixer.part.state_bytes()

    def load(self, take, p: str):
        self.mixer.load(take, p, 1, "mix.")
        if self.ffn is not None:
            self.ffn.load(take, p, 2, "mlp.")
        else:       # without the sublayer its norm and connections mean nothing
            take.drop(p + "norm2", *(f"{p}hc2.{n}" for n in ("in", "out", "mix")))

    def mix_tokens(self, h, rows, cache, state):
        proj, act = self.mixer.project_in(h)
        self.mixer.part(proj, rows, cache, state, act)
        return self.mixer.project_out(act)

    def feed_forward(self, h, counts):
        """The projected output and the routed experts' part (or None); either may be missing."""
        proj, act = self.ffn.project_in(h)
        routed = self.ffn.part(h, proj, act, counts)
        return self.ffn.project_out(act), routed


class StreamDecoder(PlanDecoder):
    def __init__(self, cfg: ModelConfig, device=None):
        if not 1 <= cfg.layer_plan.streams <= hc.MAX_STREAMS:
            raise ValueError(f"between 1 and {hc.MAX_STREAMS} residual streams are supported")
        super().__init__(cfg, device)
        self.head = _buf(torch.zeros(cfg.vocab_size, self.width_pad, dtype=self.dtype, device=device))

    @property
    def output_weight(self):
        return self.head

    def make_layer(self, index, spec, device):
        return StreamLayer(spec, self.cfg.layer_plan.streams, self.width, self.width_pad, self.cfg.rms_norm_eps, self.dtype,
                           device)

    @torch.no_grad()
    def load_tensors(self, tensors):
        """Fills the module from a Lobutar checkpoint's tensors (``embed``, ``l<i>.norm1``, ``l<i>.mix.q`` ...,
        ``l<i>.hc1.in`` ..., ``l<i>.mlp.e<j>.up`` ..., ``final.norm``, ``head``); every tensor must be there with its
        configured shape and none may be left over."""
        take = CheckpointTensors(tensors)
        put(self.embed, take("embed", self.cfg.vocab_size, self.width))
        put(self.head, take("head", self.cfg.vocab_size, self.width))
        put(self.final_gain, take("final.norm", self.width).float())
        for i, layer in enumerate(self.layers):
            layer.load(take, f"l{self.cfg.layer_plan.name(i)}.")
        take.done()
        return self

    @torch.no_grad()
    def randomize(self, seed: int = 0):
        """Random weights of the right scale (benchmarks); padding is not kept apart."""
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf == "turns":
                continue
            if leaf == "mix":
                p.copy_(torch.eye(p.shape[0]))
            elif leaf in ("read", "lam"):
                p.fill_(1.0 / p.numel() if leaf == "read" else 0.5)
            elif leaf in ("correction", "in_bias", "out_bias"):
                p.normal_(0.0, 0.01, generator=g)
            elif p.dim() == 1:
                p.fill_(1.0)
            else:
                p.normal_(0.0, 1.0 if name == "embed" else 1.0 / math.sqrt(p.shape[-1]), generator=g)
        return self

    def forward(self, rows, caches, states, final=True, record=None):
        eps, W, runs = self.cfg.rms_norm_eps, self.width, self.cfg.layer_plan.runs
        counts, at = None, 0
        experts = [self.layers[r.layer].experts for r in runs]
        if any(experts):     # cleared once per step for all runs
            counts = torch.zeros(len(runs), max(experts), dtype=torch.int32, device=self.embed.device)
        subs = [s for r in runs for s in (self.layers[r.layer].mixer, self.layers[r.layer].ffn) if s is not None]
        x, h = hc.embed_rows(rows.tokens, self.embed, self.cfg.layer_plan.streams, subs[0].read, subs[0].gain, W, eps)
        total = None

        def connect(sub, y, routed):
            """Behind a sublayer: the write, and the read in front of the next one (or the streams' sum at the end)."""
            nonlocal h, total, at
            at += 1
            if at < len(subs):
                h = hc.connect(x, y, sub.mix, sub.write, W, eps, subs[at].read, subs[at].gain, routed)
            elif final:
                h = hc.connect(x, y, sub.mix, sub.write, W, eps, None, self.final_gain, routed, keep=record is not None)
            else:
                total = torch.empty(x.shape[0], x.shape[2], dtype=torch.float32, device=x.device)
                hc.connect(x, y, sub.mix, sub.write, W, eps, None, None, routed, total=total, keep=record is not None)

        for r in runs:
            layer = self.layers[r.layer]
            connect(layer.mixer, layer.mix_tokens(h, rows, caches[r.index], states[r.index]), None)
            if layer.ffn is not None:
                n = layer.experts
                connect(layer.ffn, *layer.feed_forward(h, counts[r.index, :n] if n else None))
            if record is not None:
                record.append(x.sum(1))
        return h if final else total

"""Serving modules of decoders that are described by a layer plan (``models/layer_plan.py``): the weights of every layer
in the layout the kernels read, and the layer itself as a sequence of framework ops.  The cache, the recurrent state and
the scheduler belong to the rollout engine.

``PlanDecoder`` is what the engine talks to: per layer the cache and state it needs, and one forward over the rows of a
step.  Subclasses supply the layers and the residual stream; ``build_decoder`` picks one by the plan.  ``SandwichDecoder``
here: mixers side by side, norms before and after each sublayer, looped layers.

Layout against the checkpoint:
  * one input projection per layer, rows ``[left q | left k | right q | right k | right v | right g]``, each block's heads
    padded with zero rows to the sizes the kernels store; the 32-bit gate projections are separate;
  * the model width is padded to a multiple of 8, feed-forward widths likewise ([gate | up] rows);
  * norm gains are 32-bit and stored as the factor they multiply by (``1 + w`` for those kept around zero).
Zero padding changes no score, state or output; means are taken over the true sizes."""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch
import torch.nn as nn

from ..ops import matrix_memory as mm
from ..ops import sandwich
from ..ops import window_attention as wa
from ..ops.gemm import linear_forward
from .config import ModelConfig
from .layer_plan import ConvLayerSpec, LayerSpec, ParallelLayerSpec, StreamLayerSpec


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def _buf(t: torch.Tensor) -> nn.Parameter:
    return nn.Parameter(t, requires_grad=False)


def put(dst: torch.Tensor, t: torch.Tensor):
    """Copies ``t`` into the leading corner of ``dst``."""
    dst[tuple(slice(0, s) for s in t.shape)].copy_(t)


def put_heads(dst: torch.Tensor, t: torch.Tensor, heads: int, dim: int, pad: int):
    """[heads * dim, ...] -> rows of heads padded to ``pad``."""
    put(dst.view(heads, pad, *dst.shape[1:]), t.view(heads, dim, *t.shape[1:]))


class CheckpointTensors:
    """Tensors of a checkpoint, taken one by one: each must be there with its configured shape, none may be left over."""

    def __init__(self, tensors: Dict[str, torch.Tensor]):
        self.left = dict(tensors)

    def __call__(self, name: str, *shape: int) -> torch.Tensor:
        if name not in self.left:
            raise KeyError(f"checkpoint lacks '{name}'")
        t = self.left.pop(name)
        if tuple(t.shape) != shape:
            raise ValueError(f"'{name}' has shape {tuple(t.shape)}, the configuration says {shape}")
        return t

    def drop(self, *names: str):
        """Tensors the configuration has no use for, if they are there."""
        for n in names:
            self.left.pop(n, None)

    def done(self):
        if self.left:
            raise ValueError(f"checkpoint tensors without a place in the model: {sorted(self.left)[:8]}")


class PlanLayer(nn.Module):
    """One layer's weights and its forward over the rows of a step."""

    def __init__(self, spec: LayerSpec, width: int, width_pad: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.width, self.width_pad, self.eps = spec, width, width_pad, eps
        a, m = spec.attention, spec.memory
        self.att_dim = wa.padded_head_dim(a.dim)
        self.mem_dim, self.mem_vdim = mm.padded_key_dim(m.dim), mm.padded_value_dim(m.vdim)
        self.ffn_pad = _up(spec.ffn, 8)
        blocks = (("q", a.heads * self.att_dim), ("k", a.kv_heads * self.att_dim), ("mq", m.heads * self.mem_dim),
                  ("mk", m.heads * self.mem_dim), ("mv", m.heads * self.mem_vdim), ("mg", m.heads * self.mem_vdim))
        self.off, n = {}, 0
        for name, size in blocks:
            self.off[name] = n
            n += size
        f32 = dict(dtype=torch.float32, device=device)
        act = dict(dtype=dtype, device=device)
        self.in_proj, self.in_bias = _buf(torch.zeros(n, width_pad, **act)), _buf(torch.zeros(n, **f32))
        self.gate_w, self.gate_b = _buf(torch.zeros(2 * m.heads, width_pad, **act)), _buf(torch.zeros(2 * m.heads, **f32))
        self.att_out = _buf(torch.zeros(width_pad, a.heads * self.att_dim, **act))
        self.mem_out = _buf(torch.zeros(width_pad, m.heads * self.mem_vdim, **act))
        self.mem_gain = _buf(torch.zeros(m.heads * self.mem_vdim, **f32))
        self.slopes = _buf(torch.tensor(a.slopes(), **f32))
        names = ["pre1", "post1", "gain_att", "gain_mem"] + (["pre2", "post2"] if spec.ffn else [])
        for k in names:
            setattr(self, k, _buf(torch.zeros(width_pad, **f32)))
        if spec.ffn:
            self.fc1 = _buf(torch.zeros(2 * self.ffn_pad, width_pad, **act))
            self.fc2 = _buf(torch.zeros(width_pad, self.ffn_pad, **act))

    # ---- sizes the engine allocates by
    def cache_shape(self):
        return self.spec.attention.kv_heads, self.att_dim

    def new_state(self, slots: int, device) -> mm.MemoryState:
        return mm.MemoryState.allocate(slots, self.spec.memory.heads, self.mem_dim, self.mem_vdim, device)

    def state_bytes(self) -> int:
        return mm.MemoryState.bytes_per_slot(self.spec.memory.heads, self.mem_dim, self.mem_vdim)

    # ---- forward
    def mixers(self, h, rows, cache, state):
        """Both mixers on the same input; returns their outputs in front of the per-mixer norms."""
        a, m, off = self.spec.attention, self.spec.memory, self.off
        proj = linear_forward(h, self.in_proj, self.in_bias)
        o = wa.window_attention(proj, off["q"], off["k"], a.heads, a.kv_heads, self.att_dim, rows, cache, self.slopes,
                                a.scale, a.window)
        r = mm.matrix_memory(proj, off["mq"], off["mk"], off["mv"], off["mg"], h, self.gate_w, self.gate_b, m.gate_cap,
                             m.dim ** -0.5, m.heads, self.mem_dim, self.mem_vdim, m.vdim, rows, state, self.mem_gain,
                             self.eps)
        return linear_forward(o, self.att_out), linear_forward(r, self.mem_out)

    def forward(self, x, h, rows, cache, state, next_gain, x_add=None, step=None):
        """One run: residual ``x`` (32-bit, updated in place) and this layer's normed input ``h``; returns the next
        run's normed input.  ``x_add`` / ``step`` join the residual behind this layer (start of the next pass)."""
        ya, yb = self.mixers(h, rows, cache, state)
        pair = dict(y2=yb, gain_a=self.gain_att, gain_b=self.gain_mem)
        if not self.spec.ffn:
            return sandwich.add_sublayer(x, ya, self.post1, self.width, self.eps, next_gain, x_add, step, **pair)
        h = sandwich.add_sublayer(x, ya, self.post1, self.width, self.eps, self.pre2, **pair)
        y = linear_forward(sandwich.swiglu(linear_forward(h, self.fc1)), self.fc2)
        return sandwich.add_sublayer(x, y, self.post2, self.width, self.eps, next_gain, x_add, step)


class PlanDecoder(nn.Module):
    """Base of the decoders a layer plan describes: embedding, layers, final norm, output matrix, and the interface of the
    rollout engine."""

    def __init__(self, cfg: ModelConfig, device=None):
        super().__init__()
        self.cfg = cfg
        self.dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}.get(cfg.dtype)
        if self.dtype is None:
            raise ValueError(f"layer-plan decoders run in bfloat16 or float32, not {cfg.dtype}")
        self.width, self.width_pad = cfg.hidden_size, _up(cfg.hidden_size, 8)
        self.embed = _buf(torch.zeros(cfg.vocab_size, self.width_pad, dtype=self.dtype, device=device))
        self.layers = nn.ModuleList([self.make_layer(i, sp, device) for i, sp in enumerate(cfg.layer_plan.layers)])
        self.final_gain = _buf(torch.zeros(self.width_pad, dtype=torch.float32, device=device))

    @property
    def output_weight(self) -> torch.Tensor:
        """[vocab, width] matrix of the logits."""
        raise NotImplementedError

    def make_layer(self, index: int, spec, device) -> nn.Module:
        raise NotImplementedError

    def forward(self, rows, caches, states, final: bool = True, record: Optional[list] = None):
        """All layer runs over the rows of one step.  ``caches`` / ``states``: one per layer run.  Returns the
        final-normed hidden states of all rows, or with ``final=False`` the 32-bit residual in front of the final norm
        (``final_rows`` then norms the rows that are wanted).  ``record`` collects the residual after every run."""
        raise NotImplementedError

    def final_rows(self, x, rows=None):
        return sandwich.norm_rows(x, self.final_gain, self.width, self.cfg.rms_norm_eps, self.embed.dtype, rows)

    # ---- what the engine allocates for every layer run
    def new_caches(self, blocks: int, block_size: int, device) -> list:
        """Paged cache of every run, one row (of any shape) per token; None for runs without one."""
        shapes = [self.layers[r.layer].cache_shape() for r in self.cfg.layer_plan.runs]
        return [torch.zeros(blocks, block_size, *s, dtype=self.dtype, device=device) if s else None for s in shapes]

    def new_states(self, slots: int, device) -> list:
        """Recurrent state of every run, one per request slot; None for runs without one."""
        return [self.layers[r.layer].new_state(slots, device) for r in self.cfg.layer_plan.runs]

    def cache_bytes_per_token(self) -> int:
        shapes = [self.layers[r.layer].cache_shape() for r in self.cfg.layer_plan.runs]
        return sum(math.prod(s) for s in shapes if s) * self.embed.element_size()

    def state_bytes_per_slot(self) -> int:
        return sum(self.layers[r.layer].state_bytes() for r in self.cfg.layer_plan.runs)


class SandwichDecoder(PlanDecoder):
    def __init__(self, cfg: ModelConfig, device=None):
        super().__init__(cfg, device)
        plan, f32 = cfg.layer_plan, dict(dtype=torch.float32, device=device)
        act = dict(dtype=self.dtype, device=device)
        self.pos_table = _buf(torch.zeros(cfg.max_position_embeddings, self.width_pad, **act))
        self.loop_step = _buf(torch.zeros(plan.loop_times, self.width_pad, **f32)) if plan.loop_times else None
        self.head = _buf(torch.zeros(cfg.vocab_size, self.width_pad, **act))

    @property
    def output_weight(self):
        return self.head

    def make_layer(self, index, spec, device):
        return PlanLayer(spec, self.width, self.width_pad, self.cfg.rms_norm_eps, self.dtype, device)

    # ------------------------------------------------------------------ checkpoint
    @torch.no_grad()
    def load_tensors(self, tensors: Dict[str, torch.Tensor]):
        """Fills the module from a Nafitar checkpoint's tensors (``embed``, ``pos``, ``loop.step``, ``l<i>.norm1``,
        ``l<i>.mix.left.q`` ..., ``final.norm``, ``head``); every tensor must be there with its configured shape and
        none may be left over."""
        take, W = CheckpointTensors(tensors), self.width
        put(self.embed, take("embed", self.cfg.vocab_size, W))
        put(self.pos_table, take("pos", self.cfg.max_position_embeddings, W))
        put(self.head, take("head", self.cfg.vocab_size, W))
        put(self.final_gain, 1 + take("final.norm", W).float())
        if self.loop_step is not None:
            put(self.loop_step, take("loop.step", self.loop_step.shape[0], W).float())
        for i, ly in enumerate(self.layers):
            a, m, o = ly.spec.attention, ly.spec.memory, ly.off
            p, D, dk, dv = f"l{i}.", ly.att_dim, ly.mem_dim, ly.mem_vdim
            put(ly.pre1, 1 + take(p + "norm1", W).float())
            put(ly.post1, 1 + take(p + "norm1b", W).float())
            for key, nm, n, dim, pad in (("q", "left.q", a.heads, a.dim, D), ("k", "left.k", a.kv_heads, a.dim, D),
                                         ("mq", "right.q", m.heads, m.dim, dk), ("mk", "right.k", m.heads, m.dim, dk),
                                         ("mv", "right.v", m.heads, m.vdim, dv), ("mg", "right.g", m.heads, m.vdim, dv)):
                put_heads(ly.in_proj[o[key]:o[key] + n * pad], take(p + "mix." + nm, n * dim, W), n, dim, pad)
                if key in ("q", "k"):
                    put_heads(ly.in_bias[o[key]:o[key] + n * pad], take(p + f"mix.{nm}.b", n * dim), n, dim, pad)
            for r, nm in enumerate(("right.i", "right.f")):
                put(ly.gate_w[r * m.heads:(r + 1) * m.heads], take(p + "mix." + nm, m.heads, W))
                put(ly.gate_b[r * m.heads:(r + 1) * m.heads], take(p + f"mix.{nm}.b", m.heads).float())
            for dst, nm, n, dim, pad in ((ly.att_out, "left.o", a.heads, a.dim, D), (ly.mem_out, "right.o", m.heads, m.vdim, dv)):
                put(dst.view(dst.shape[0], n, pad), take(p + "mix." + nm, W, n * dim).view(W, n, dim))
            put_heads(ly.mem_gain, take(p + "mix.right.norm", m.heads * m.vdim).float(), m.heads, m.vdim, dv)
            put(ly.gain_att, take(p + "mix.left.out", W).float())
            put(ly.gain_mem, take(p + "mix.right.out", W).float())
            if ly.spec.ffn:
                f = ly.spec.ffn
                put(ly.pre2, 1 + take(p + "norm2", W).float())
                put(ly.post2, 1 + take(p + "norm2b", W).float())
                put(ly.fc1[:f], take(p + "mlp.gate", f, W))
                put(ly.fc1[ly.ffn_pad:ly.ffn_pad + f], take(p + "mlp.up", f, W))
                put(ly.fc2, take(p + "mlp.down", W, f))
        take.done()
        return self

    @torch.no_grad()
    def randomize(self, seed: int = 0):
        """Random weights of the right scale (benchmarks); gains stay near one, padding is not kept apart."""
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if name.endswith("slopes"):
                continue
            if p.dim() == 1:
                p.fill_(0.0 if name.endswith(("in_bias", "gate_b")) else 1.0)
            else:
                p.normal_(0.0, 0.3 if name in ("pos_table", "loop_step") else
                          1.0 if name == "embed" else 1.0 / math.sqrt(p.shape[1]), generator=g)
        return self

    # ------------------------------------------------------------------ forward
    def forward(self, rows, caches, states, final: bool = True, record: Optional[list] = None):
        plan, eps = self.cfg.layer_plan, self.cfg.rms_norm_eps
        runs = plan.runs
        opens = [r.opens_pass for r in runs] + [None]
        step = self.loop_step[0] if opens[0] is not None else None
        x, first, h = sandwich.embed_rows(rows.tokens, rows.pos, self.embed, self.pos_table, self.layers[runs[0].layer].pre1,
                                          self.width, eps, step, keep_first=plan.loop_times > 1)
        for r in runs:
            t = opens[r.index + 1]
            last = r.index + 1 == len(runs)
            gain = (self.final_gain if final else None) if last else self.layers[runs[r.index + 1].layer].pre1
            layer = self.layers[r.layer]
            if record is None or t is None:
                h = layer(x, h, rows, caches[r.index], states[r.index], gain, first if t else None,
                          self.loop_step[t] if t is not None else None)
                if record is not None:
                    record.append(x.clone())
            else:   # the recorded residual is the one in front of what opens the next pass
                layer(x, h, rows, caches[r.index], states[r.index], None)
                record.append(x.clone())
                x += self.loop_step[t] + (first if t else 0)
                h = sandwich.norm_rows(x, gain, self.width, eps, self.embed.dtype)
        return h if final else x


def build_decoder(cfg: ModelConfig, device=None) -> PlanDecoder:
    """The serving module of a layer-plan configuration."""
    from .conv_decoder import ConvDecoder
    from .parallel_decoder import ParallelDecoder
    from .stream_decoder import StreamDecoder
    cls = {ParallelLayerSpec: ParallelDecoder, StreamLayerSpec: StreamDecoder, LayerSpec: SandwichDecoder,
           ConvLayerSpec: ConvDecoder}
    return cls[type(cfg.layer_plan.layers[0])](cfg, device)

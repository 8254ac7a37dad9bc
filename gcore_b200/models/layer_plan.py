"""Per-layer architecture description for decoders whose layers differ from one another and may run more than once.

The families of ``ModelConfig`` that came first describe all layers with one set of numbers.  A *layer plan* lists the
layers one by one - which mixers a layer runs, the size of each, its feed-forward - and may loop a range of layers with
shared weights.  Every run of a layer (a looped layer counts once per pass) owns its cache and state, so the serving engine
sizes both from ``LayerPlan.runs``.

Two kinds of layer are described: ``LayerSpec`` (two mixers side by side, then a feed-forward, norms before and after each)
and ``ParallelLayerSpec`` (one mixer and a feed-forward that read the same normed input)."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple, Union


@dataclass(frozen=True)
class WindowAttentionSpec:
    """Grouped-query softmax attention over a sliding window: position i sees j with ``0 <= i - j < window``; the score
    is ``(q . k) * scale - slope_h * (i - j)``.  The values are the keys (one cached row serves both)."""
    heads: int
    kv_heads: int
    dim: int
    window: int
    scale: float

    def __post_init__(self):
        if self.heads < 1 or self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError("query heads must be a positive multiple of the key/value heads")
        if self.window < 1 or self.dim < 1:
            raise ValueError("attention window and head size must be positive")

    def slopes(self) -> List[float]:
        """Distance penalty per head: a geometric series that ends at 2^-8."""
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Recurrent matrix memory with exponential input gate and a running-maximum stabiliser (mLSTM): per head a
    ``dim x vdim`` state, a ``dim`` normaliser and a scalar maximum, all in 32-bit."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1 or not self.gate_cap > 0:
            raise ValueError("matrix-memory sizes and the gate cap must be positive")


@dataclass(frozen=True)
class LayerSpec:
    """One layer: an attention and a recurrent mixer that read the same input side by side, and a gated feed-forward
    (``ffn`` = 0: none)."""
    attention: WindowAttentionSpec
    memory: MatrixMemorySpec
    ffn: int = 0


@dataclass(frozen=True)
class YarnSpec:
    """Context extension of a rotation: pairs that turn fewer than ``slow`` times over ``original`` positions are slowed
    down by ``factor``, those that turn more than ``fast`` times keep their frequency, the ones between are blended."""
    factor: float
    original: float
    fast: float
    slow: float

    def __post_init__(self):
        if min(self.factor, self.original, self.fast, self.slow) <= 0:
            raise ValueError("rotation scaling needs positive constants")


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of ``dims`` dimensions, neighbours paired (2i with 2i + 1), angle = position * base^(-2i/dims)."""
    dims: int
    base: float
    scaling: Optional[YarnSpec] = None

    def __post_init__(self):
        if self.dims < 2 or self.dims % 2 or self.base <= 1:
            raise ValueError("a rotation needs an even number of dimensions and a base above 1")

    def frequencies(self) -> List[float]:
        n, sc = self.dims, self.scaling
        freq = [self.base ** (-2.0 * i / n) for i in range(n // 2)]
        if sc is None:
            return freq

        def pair_of(turns):
            return n * math.log(sc.original / (2 * math.pi * turns)) / (2 * math.log(self.base))

        lo, hi = max(math.floor(pair_of(sc.fast)), 0), min(math.ceil(pair_of(sc.slow)), n - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)]
        return [f / sc.factor * r + f * (1 - r) for f, r in zip(freq, ramp)]

    def magnitude(self) -> float:
        """Factor of both cosine and sine."""
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling.factor) + 1.0


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Causal softmax attention over a cached latent: per token one normed vector of ``kv_rank`` that every head expands to
    its own key (``dim``) and value (``vdim``), and one rotated key part of ``rot_dim`` that all heads share; the output of
    a head is scaled by a sigmoid gate."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotarySpec

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.kv_rank) < 1:
            raise ValueError("latent-attention sizes must be positive")
        if self.rot.dims != self.rot_dim:
            raise ValueError("the rotation must cover the rotated key part")


@dataclass(frozen=True)
class RetentionSpec:
    """Linear attention with one fixed decay per head: a ``dim x vdim`` state per head in 32-bit."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1 or len(self.decay) != self.heads:
            raise ValueError("retention needs positive sizes and one decay per head")
        if not all(0 <= d <= 1 for d in self.decay):
            raise ValueError("retention decays must lie in [0, 1]")


@dataclass(frozen=True)
class DenseSpec:
    """Gated feed-forward: ``down(silu(gate h) * up h)``."""
    ff: int


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture of small feed-forwards ``down(relu(up h)^2)``: softmax scores, chosen with a correction that the weights do
    not carry, and a shared expert (``shared_ff`` = 0: none) behind a sigmoid gate of one number per token."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0

    def __post_init__(self):
        if not 1 <= self.top <= self.experts or self.ff < 1 or self.shared_ff < 0:
            raise ValueError("experts need positive sizes and at most as many choices as experts")


@dataclass(frozen=True)
class ParallelLayerSpec:
    """One layer whose mixer and feed-forward (None: none) read the same normed input."""
    mixer: Union[LatentAttentionSpec, RetentionSpec]
    ffn: Union[DenseSpec, ExpertsSpec, None] = None


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``index`` numbers the runs (= the cache / state set), ``layer`` names the weights.
    ``opens_pass`` is the pass number when this run is the first of a pass of the loop, else None."""
    index: int
    layer: int
    opens_pass: Optional[int] = None


@dataclass(frozen=True)
class LayerPlan:
    layers: Tuple[Union[LayerSpec, ParallelLayerSpec], ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0          # 0: no loop

    def __post_init__(self):
        if not self.layers:
            raise ValueError("a layer plan needs at least one layer")
        if self.loop_times < 0 or (self.loop_times and not 0 <= self.loop_start < self.loop_stop <= len(self.layers)):
            raise ValueError("the looped layers must be a non-empty range of the layer list")

    @property
    def runs(self) -> List[LayerRun]:
        order: List[Tuple[int, Optional[int]]] = []
        if self.loop_times:
            order += [(i, None) for i in range(self.loop_start)]
            for t in range(self.loop_times):
                order += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
            order += [(i, None) for i in range(self.loop_stop, len(self.layers))]
        else:
            order = [(i, None) for i in range(len(self.layers))]
        return [LayerRun(n, i, t) for n, (i, t) in enumerate(order)]


def _need(d: Dict[str, Any], key: str, where: str):
    if key not in d:
        raise ValueError(f"{where} lacks '{key}'")
    return d[key]


def nafitar_plan(conf: Dict[str, Any]) -> LayerPlan:
    """Layer plan of a Nafitar ``config.json``."""
    layers = []
    for i, entry in enumerate(_need(conf, "layers", "config")):
        where = f"layers[{i}]"
        if entry.get("type") != "parallel":
            raise ValueError(f"{where}: unknown mixer type {entry.get('type')!r}")
        left, right = entry["mixer"]["left"], entry["mixer"]["right"]
        att = WindowAttentionSpec(heads=left["heads"], kv_heads=left["kv_heads"], dim=left["dim"],
                                  window=left["mask"]["size"], scale=float(left["scale"]))
        if left.get("vdim", att.dim) != att.dim:
            raise ValueError(f"{where}: the values are the keys, so 'vdim' must equal 'dim'")
        mem = MatrixMemorySpec(heads=right["heads"], dim=right["dim"], vdim=right["vdim"],
                               gate_cap=float(right["gate_cap"]))
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"{where}: unknown feed-forward kind {mlp.get('kind')!r}")
        layers.append(LayerSpec(att, mem, mlp["ff"] if mlp is not None else 0))
    loop = conf.get("loop")
    if loop:
        return LayerPlan(tuple(layers), loop["start"], loop["stop"], loop["times"])
    return LayerPlan(tuple(layers))


def _rotation(d: Dict[str, Any], where: str) -> RotarySpec:
    sc = d.get("scaling")
    yarn = YarnSpec(*(float(_need(sc, k, where + ".scaling")) for k in ("factor", "original", "fast", "slow"))) if sc else None
    return RotarySpec(dims=_need(d, "dims", where), base=float(_need(d, "base", where)), scaling=yarn)


def _latent_attention(m: Dict[str, Any], where: str) -> LatentAttentionSpec:
    return LatentAttentionSpec(rot=_rotation(_need(m, "rot", where), where + ".rot"), scale=float(_need(m, "scale", where)),
                               **{k: _need(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")})


def _retention(m: Dict[str, Any], where: str) -> RetentionSpec:
    return RetentionSpec(decay=tuple(float(x) for x in _need(m, "decay", where)),
                         **{k: _need(m, k, where) for k in ("heads", "dim", "vdim")})


MIXER_READERS = {"latent_attention": _latent_attention, "retention": _retention}


def _feed_forward(m: Optional[Dict[str, Any]], where: str):
    if m is None:
        return None
    kind = m.get("kind")
    if kind == "dense":
        return DenseSpec(_need(m, "ff", where))
    if kind != "moe":
        raise ValueError(f"{where}: unknown feed-forward kind {kind!r}")
    router, shared = _need(m, "router", where), m.get("shared")
    return ExpertsSpec(experts=_need(router, "experts", where), top=_need(router, "top", where),
                       ff=_need(_need(m, "expert", where), "ff", where), shared_ff=shared["ff"] if shared else 0)


def kedesun_plan(conf: Dict[str, Any]) -> LayerPlan:
    """Layer plan of a Kedesun ``config.json``."""
    layers = []
    for i, entry in enumerate(_need(conf, "layers", "config")):
        where = f"layers[{i}]"
        reader = MIXER_READERS.get(entry.get("type"))
        if reader is None:
            raise ValueError(f"{where}: unknown mixer type {entry.get('type')!r}")
        layers.append(ParallelLayerSpec(reader(_need(entry, "mixer", where), where + ".mixer"),
                                        _feed_forward(entry.get("mlp"), where + ".mlp")))
    return LayerPlan(tuple(layers))

"""Per-layer architecture description for decoders whose layers differ from one another and may run more than once.

The families of ``ModelConfig`` that came first describe all layers with one set of numbers.  A *layer plan* lists the
layers one by one - which mixers a layer runs, the size of each, its feed-forward - and may loop a range of layers with
shared weights.  Every run of a layer (a looped layer counts once per pass) owns its cache and state, so the serving engine
sizes both from ``LayerPlan.runs``.

Four kinds of layer are described: ``LayerSpec`` (two mixers side by side, then a feed-forward, norms before and after
each), ``ParallelLayerSpec`` (one mixer and a feed-forward that read the same normed input), ``StreamLayerSpec`` (a mixer,
then a feed-forward, each reading a mixture of several residual streams and writing to all of them) and ``ConvLayerSpec`` (one
mixer or a weighted sum of several, then a feed-forward, each behind a norm and a short convolution over time)."""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
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
    """Rotation of ``dims`` dimensions, angle = position * base^(-2i/dims) / ``slow``.  Pair i is two neighbours (2i with
    2i + 1) or, with ``halves``, dimension i and dimension i + dims/2."""
    dims: int
    base: float
    scaling: Optional[YarnSpec] = None
    slow: float = 1.0
    halves: bool = False

    def __post_init__(self):
        if self.dims < 2 or self.dims % 2 or self.base <= 1 or self.slow <= 0:
            raise ValueError("a rotation needs an even number of dimensions, a base above 1 and a positive scaling")

    def neighbours(self, dim: int) -> List[int]:
        """Order of a head's ``dim`` dimensions in which pair i is 2i with 2i + 1.  Applied to queries and keys alike it
        changes neither their products nor their norms."""
        n = self.dims
        turned = [i // 2 + (i % 2) * (n // 2) for i in range(n)] if self.halves else list(range(n))
        return turned + list(range(n, dim))

    def frequencies(self) -> List[float]:
        n, sc = self.dims, self.scaling
        freq = [self.base ** (-2.0 * i / n) / self.slow for i in range(n // 2)]
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
    its own key (``dim``) and value (``vdim``), and one rotated key part of ``rot_dim`` that all heads share.  ``window``:
    position i sees j with ``0 <= i - j < window`` (0: every j <= i); ``sink``: a learned logit per head joins the softmax
    denominator; ``gate``: the output is scaled by sigmoids, one per "head" or one per "element"."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    window: int = 0
    sink: bool = False
    gate: str = "head"

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.kv_rank) < 1 or self.window < 0:
            raise ValueError("latent-attention sizes must be positive")
        if self.gate not in ("head", "element"):
            raise ValueError(f"unknown output gate {self.gate!r}")
        if self.rot.dims != self.rot_dim:
            raise ValueError("the rotation must cover the rotated key part")


@dataclass(frozen=True)
class DifferentialAttentionSpec:
    """Grouped-query causal attention whose heads subtract two softmax maps over the same values: per head two queries and
    per key/value head two keys of ``dim``, the first ``rot.dims`` of them rotated; the difference ``a1 - lambda * a2`` is
    normed over the head's ``vdim`` values, scaled by ``1 - diff`` and by a sigmoid gate of the head.  lambda is learned
    (four vectors of ``dim``) around ``diff``.  The projections have biases."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: RotarySpec

    def __post_init__(self):
        if self.heads < 1 or self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError("query heads must be a positive multiple of the key/value heads")
        if min(self.dim, self.vdim) < 1 or self.rot.dims > self.dim:
            raise ValueError("attention sizes must be positive and hold the rotated dimensions")


@dataclass(frozen=True)
class ScoredAttentionSpec:
    """Grouped-query attention with a bias on every score.  Queries and keys may be rotated (``rot``) and then divided by
    their root mean square (``unit``).  ``weights``: "softmax" of the scores, or "sigmoid" of each, not normalised over the
    keys.  ``distance``: two learned numbers per head take ``r1 * ln(1 + r2 * (i - j))`` off a score; ``head_bias``: a learned
    number per head is added to it.  ``window`` (0: none): position i sees j with ``0 <= i - j < window``, and the first
    ``keep`` positions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    weights: str = "softmax"
    rot: Optional[RotarySpec] = None
    unit: bool = False
    distance: bool = False
    head_bias: bool = False
    window: int = 0
    keep: int = 0

    def __post_init__(self):
        if self.heads < 1 or self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError("query heads must be a positive multiple of the key/value heads")
        if min(self.dim, self.vdim) < 1 or (self.rot is not None and self.rot.dims > self.dim):
            raise ValueError("attention sizes must be positive and hold the rotated dimensions")
        if min(self.window, self.keep) < 0:
            raise ValueError("a window and its kept positions must not be negative")
        if self.weights not in ("softmax", "sigmoid"):
            raise ValueError(f"unknown attention weights {self.weights!r}")


@dataclass(frozen=True)
class RetentionSpec:
    """Linear attention with one fixed decay per head: a ``dim x vdim`` state per head in 32-bit.  Queries and keys may be
    rotated (``rot``); ``act``: "silu" on queries, keys and values, or "".  The output is normed per "head" or over all heads
    together ("joint", with a gain), and gated by a "silu" or "sigmoid"; ``scale``: factor of a query-key product."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    scale: Optional[float] = None        # default: dim^-1/2
    rot: Optional[RotarySpec] = None
    act: str = ""
    norm: str = "head"
    gate: str = "silu"

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1 or len(self.decay) != self.heads:
            raise ValueError("retention needs positive sizes and one decay per head")
        if not all(0 <= d <= 1 for d in self.decay):
            raise ValueError("retention decays must lie in [0, 1]")
        if self.act not in ("", "silu") or (self.norm, self.gate) not in (("head", "silu"), ("joint", "sigmoid")):
            raise ValueError(f"unknown retention activation {self.act!r}, norm {self.norm!r} or gate {self.gate!r}")
        if self.rot is not None and (self.rot.dims > self.dim or self.act):
            raise ValueError("rotated dimensions must lie in the head, and go without an activation")

    def product_scale(self) -> float:
        return self.dim ** -0.5 if self.scale is None else self.scale


@dataclass(frozen=True)
class DenseSpec:
    """Feed-forward: ``down(silu(gate h) * up h)`` ("silu_gate") or ``down(relu(up h)^2)`` ("relu2")."""
    ff: int
    act: str = "silu_gate"


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture of small feed-forwards, ``down(relu(up h)^2)`` ("relu2") or ``down(silu(gate h) * up h)`` ("silu_gate").  The
    ``top`` experts are chosen by score + correction; the weights carry the scores alone, normalised or not, times
    ``scale``.  Scores are a softmax or sigmoids of the router's logits.  With ``groups`` > 1 only experts of the ``keep``
    groups of neighbours with the largest sum of two best choice scores take part.  A shared expert (``shared_ff`` = 0:
    none) runs for every token, behind a sigmoid gate of one number per token if ``shared_gate``."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    act: str = "relu2"
    score: str = "softmax"
    normalize: bool = True
    scale: float = 1.0
    groups: int = 1
    keep: int = 1
    shared_gate: bool = True

    def __post_init__(self):
        if not 1 <= self.top <= self.experts or self.ff < 1 or self.shared_ff < 0:
            raise ValueError("experts need positive sizes and at most as many choices as experts")
        if self.act not in ("relu2", "silu_gate") or self.score not in ("softmax", "sigmoid"):
            raise ValueError(f"unknown expert activation {self.act!r} or score {self.score!r}")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError("expert groups must be equal and some of them kept")
        if self.top > self.experts // self.groups * self.keep:
            raise ValueError("the kept groups hold fewer experts than are chosen")


@dataclass(frozen=True)
class ParallelLayerSpec:
    """One layer whose mixer and feed-forward (None: none) read the same normed input."""
    mixer: Union[LatentAttentionSpec, RetentionSpec]
    ffn: Union[DenseSpec, ExpertsSpec, None] = None


@dataclass(frozen=True)
class StreamLayerSpec:
    """One layer of a decoder with several residual streams (hyper-connections): a mixer, then a feed-forward (None: none),
    each behind its own norm."""
    mixer: Union[LatentAttentionSpec, DifferentialAttentionSpec]
    ffn: Union[DenseSpec, ExpertsSpec, None] = None


@dataclass(frozen=True)
class ConvLayerSpec:
    """One layer: the sum of ``mixers`` times their ``scales``, then a feed-forward (None: none), each behind a norm and a short
    causal convolution over time."""
    mixers: Tuple[Union[ScoredAttentionSpec, RetentionSpec], ...]
    scales: Tuple[float, ...]
    ffn: Optional[DenseSpec] = None

    def __post_init__(self):
        if not self.mixers or len(self.mixers) != len(self.scales):
            raise ValueError("a layer needs a mixer, and one scale per mixer")


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``index`` numbers the runs (= the cache / state set), ``layer`` names the weights.
    ``opens_pass`` is the pass number when this run is the first of a pass of the loop, else None."""
    index: int
    layer: int
    opens_pass: Optional[int] = None


@dataclass(frozen=True)
class LayerPlan:
    """``layers``: the layers that own weights.  They run in order, with a looped range, or, with ``order``, as it lists them
    (a layer may run any number of times).  ``names``: the layers' numbers in the checkpoint when they are not 0, 1, ..."""
    layers: Tuple[Union[LayerSpec, ParallelLayerSpec, StreamLayerSpec, ConvLayerSpec], ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0          # 0: no loop
    order: Tuple[int, ...] = ()
    names: Tuple[int, ...] = ()
    streams: int = 0             # residual streams of a decoder with hyper-connections
    taps: int = 0                # taps of the convolution in front of every sublayer
    residual_mult: float = 1.0   # factor of what a sublayer adds to the residual
    logit_scale: float = 1.0

    def __post_init__(self):
        if not self.layers:
            raise ValueError("a layer plan needs at least one layer")
        if self.loop_times < 0 or (self.loop_times and not 0 <= self.loop_start < self.loop_stop <= len(self.layers)):
            raise ValueError("the looped layers must be a non-empty range of the layer list")
        if self.order and (self.loop_times or not all(0 <= i < len(self.layers) for i in self.order)):
            raise ValueError("the order of a plan's runs names layers of the plan and goes without a loop")
        if self.names and len(self.names) != len(self.layers):
            raise ValueError("a plan's layer names must cover its layers")

    def name(self, i: int) -> int:
        """Number of layer i in the checkpoint."""
        return self.names[i] if self.names else i

    def windows(self) -> List[int]:
        """Distinct attention windows of the latent mixers (0: unlimited)."""
        mixers = [getattr(sp, "mixer", None) for sp in self.layers]
        return sorted({m.window for m in mixers if isinstance(m, LatentAttentionSpec)})

    @property
    def runs(self) -> List[LayerRun]:
        order: List[Tuple[int, Optional[int]]] = []
        if self.order:
            order = [(i, None) for i in self.order]
        elif self.loop_times:
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


def _differential_attention(m: Dict[str, Any], where: str) -> DifferentialAttentionSpec:
    return DifferentialAttentionSpec(rot=_rotation(_need(m, "rot", where), where + ".rot"),
                                     **{k: float(_need(m, k, where)) for k in ("scale", "diff")},
                                     **{k: _need(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")})


def _window_latent_attention(m: Dict[str, Any], where: str) -> LatentAttentionSpec:
    window = _need(_need(m, "mask", where), "size", where + ".mask")
    if window < 1:
        raise ValueError(f"{where}.mask: the window must be positive")
    return replace(_latent_attention(m, where), window=window, sink=True, gate="element")


STREAM_MIXER_READERS = {"attention": _differential_attention, "latent_attention": _window_latent_attention}


def _grouped_experts(m: Optional[Dict[str, Any]], where: str):
    """Feed-forward of a stream layer: experts are gated, with sigmoid scores that are not normalised."""
    spec = _feed_forward(m, where)
    if not isinstance(spec, ExpertsSpec):
        return spec
    router = m["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    return replace(spec, act="silu_gate", score="sigmoid", normalize=False, scale=float(router.get("scale", 1.0)),
                   groups=_need(groups, "count", where + ".router.groups"),
                   keep=_need(groups, "keep", where + ".router.groups"), shared_gate=False)


def lobutar_plan(conf: Dict[str, Any]) -> LayerPlan:
    """Layer plan of a Lobutar ``config.json``.  Entries with ``weights_of`` run another entry's layer once more."""
    entries = _need(conf, "layers", "config")
    owner = []
    for i, entry in enumerate(entries):
        j, seen = i, set()
        while entries[j].get("weights_of") is not None:
            seen.add(j)
            j = entries[j]["weights_of"]
            if not 0 <= j < len(entries) or j in seen:
                raise ValueError(f"layers[{i}]: 'weights_of' names no layer with weights")
        owner.append(j)
    names = [i for i, j in enumerate(owner) if i == j]
    layers = []
    for i in names:
        where, entry = f"layers[{i}]", entries[i]
        reader = STREAM_MIXER_READERS.get(entry.get("type"))
        if reader is None:
            raise ValueError(f"{where}: unknown mixer type {entry.get('type')!r}")
        layers.append(StreamLayerSpec(reader(_need(entry, "mixer", where), where + ".mixer"),
                                      _grouped_experts(entry.get("mlp"), where + ".mlp")))
    streams = _need(conf, "streams", "config")
    if streams < 1:
        raise ValueError("a decoder needs at least one residual stream")
    return LayerPlan(tuple(layers), order=tuple(names.index(j) for j in owner), names=tuple(names), streams=streams)


def _halves_rotation(d: Dict[str, Any], where: str) -> RotarySpec:
    sc = d.get("scaling")
    return RotarySpec(dims=_need(d, "dims", where), base=float(_need(d, "base", where)), halves=True,
                      slow=float(_need(sc, "factor", where + ".scaling")) if sc else 1.0)


def _distance_attention(m: Dict[str, Any], where: str) -> ScoredAttentionSpec:
    mask = _need(m, "mask", where)
    if _need(mask, "size", where + ".mask") < 1:
        raise ValueError(f"{where}.mask: the window must be positive")
    return ScoredAttentionSpec(distance=True, window=mask["size"], keep=_need(mask, "keep_first", where + ".mask"),
                               scale=float(_need(m, "scale", where)),
                               **{k: _need(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")})


def _sigmoid_attention(m: Dict[str, Any], where: str) -> ScoredAttentionSpec:
    return ScoredAttentionSpec(weights="sigmoid", unit=True, head_bias=True, scale=float(_need(m, "scale", where)),
                               rot=_halves_rotation(_need(m, "rot", where), where + ".rot"),
                               **{k: _need(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")})


def _conv_mixers(kind: str, m: Dict[str, Any], where: str):
    """Mixers of a layer of ``kind`` and their scales."""
    if kind == "attention":
        return (_distance_attention(m, where),), (1.0,)
    if kind == "lightning":
        return (replace(_retention(m, where), scale=1.0, act="silu", norm="joint", gate="sigmoid"),), (1.0,)
    if kind != "parallel":
        raise ValueError(f"{where}: unknown mixer type {kind!r}")
    left, right = _need(m, "left", where), _need(m, "right", where)
    turned = replace(_retention(right, where + ".right"),
                     rot=_halves_rotation(_need(right, "rot", where + ".right"), where + ".right.rot"))
    return (_sigmoid_attention(left, where + ".left"), turned), tuple(float(_need(m, k, where))
                                                                      for k in ("left_scale", "right_scale"))


def rezulorn_plan(conf: Dict[str, Any]) -> LayerPlan:
    """Layer plan of a Rezulorn ``config.json``."""
    layers = []
    for i, entry in enumerate(_need(conf, "layers", "config")):
        where = f"layers[{i}]"
        ffn = _feed_forward(entry.get("mlp"), where + ".mlp")
        if ffn is not None and not isinstance(ffn, DenseSpec):
            raise ValueError(f"{where}.mlp: unknown feed-forward kind {entry['mlp'].get('kind')!r}")
        layers.append(ConvLayerSpec(*_conv_mixers(entry.get("type"), _need(entry, "mixer", where), where + ".mixer"),
                                    replace(ffn, act="relu2") if ffn is not None else None))
    taps = _need(_need(conf, "canon", "config"), "taps", "canon")
    if taps < 1:
        raise ValueError("the input convolution needs at least one tap")
    return LayerPlan(tuple(layers), taps=taps, **{k: float(_need(conf, k, "config")) for k in ("residual_mult", "logit_scale")})


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

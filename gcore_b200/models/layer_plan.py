"""Per-layer architecture description for decoders whose layers differ from one another and may run more than once.

The families of ``ModelConfig`` that came first describe all layers with one set of numbers.  A *layer plan* lists the
layers one by one - which mixers a layer runs side by side, the size of each, its feed-forward - and may loop a range of
layers with shared weights.  Every run of a layer (a looped layer counts once per pass) owns its cache and state, so the
serving engine sizes both from ``LayerPlan.runs``."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple


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
class LayerRun:
    """One execution of a layer: ``index`` numbers the runs (= the cache / state set), ``layer`` names the weights.
    ``opens_pass`` is the pass number when this run is the first of a pass of the loop, else None."""
    index: int
    layer: int
    opens_pass: Optional[int] = None


@dataclass(frozen=True)
class LayerPlan:
    layers: Tuple[LayerSpec, ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0          # 0: no loop

    def __post_init__(self):
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

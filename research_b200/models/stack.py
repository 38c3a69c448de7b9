"""Configuration of models that are described layer by layer.

``ModelConfig`` holds one set of sizes for the whole model. A ``LayerStackConfig`` instead lists its layers; each names
the mixer it uses (with that layer's own sizes, window and rotation) and its feed-forward, or none. Mixers and
feed-forwards are small value types that know their ``config.json`` form and their tensors. Which of them a design has, and how
a layer is put together around them (norms, residual, head), is a row of ``DESIGNS``.

``config.json`` form::

    {"architecture": "Lulezen", "vocab": V, "width": d, "norm": {"eps": e}, "logit_softcap": c,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", ...} or null}, ...]}

``type`` and ``kind`` are names within a design: ``Design.mixers`` and ``Design.feed_forwards`` say what they stand for.

Tensors are named ``embed``, ``l<i>.norm1`` / ``.mix.*`` / ``.mlp.*``, ``final.norm``; matrices are stored ``[out, in]``.
Post-norm designs add ``.norm1.b`` / ``.ls1`` (and ``norm2`` / ``norm2.b`` / ``ls2`` for the feed-forward) and
``final.norm.b``; sandwich designs have ``.norm1`` / ``.norm1b`` around the mixer and ``.norm2`` / ``.norm2b`` around the feed-forward, with a
bounded norm each of them (and ``final.norm``) comes with ``.alpha`` (a scalar) and ``.b``; designs without tied embeddings have ``head``; looped stacks have ``loop.in``; stacks with a per-layer token
input have ``side.embed`` and ``l<i>.side.gate`` / ``.proj`` / ``.norm``.
"""

from __future__ import annotations

import json
import math
from collections.abc import Mapping
from dataclasses import asdict, dataclass, replace
from functools import partial
from pathlib import Path
from typing import Callable


NO_WINDOW = 1 << 30          # a window nothing reaches: plain causal attention


@dataclass(frozen=True)
class BandScaling:
    """Long waves slowed by ``factor``, short ones kept, a blend in between: with the wavelength ``l = 2 pi / f``, frequencies of
    ``l < original/high`` stay, those of ``l > original/low`` are divided, the others are mixed linearly in ``original/l``."""

    factor: float
    low: float
    high: float
    original: float

    amplitude = 1.0

    def frequencies(self, rot: "RotarySpec") -> list[float]:
        out = []
        for f in rot.plain_frequencies():
            turns = self.original * f / (2 * math.pi)          # of one wave over the original context
            keep = 1.0 if turns > self.high else 0.0 if turns < self.low else (turns - self.low) / (self.high - self.low)
            out.append(f * (keep + (1 - keep) / self.factor))
        return out


@dataclass(frozen=True)
class YarnScaling:
    """YaRN: channels that turn more than ``fast`` times over the ``original`` context keep their frequency, those below
    ``slow`` turns are divided by ``factor``, a linear ramp over the channels between; cos and sin are scaled by ``amplitude``."""

    factor: float
    original: float
    fast: float
    slow: float

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1

    def frequencies(self, rot: "RotarySpec") -> list[float]:
        def channel(turns: float) -> float:
            return rot.dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(rot.base))

        lo, hi = max(math.floor(channel(self.fast)), 0), min(math.ceil(channel(self.slow)), rot.dims - 1)
        ramps = (min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(rot.dims // 2))
        return [f * (1 - r + r / self.factor) for f, r in zip(rot.plain_frequencies(), ramps)]


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of pairs of the first ``dims`` channels by ``position * base^(-2i/dims)``: channels ``(i, i + dims/2)``, or
    ``(2i, 2i+1)`` when ``interleaved``; ``scaling`` changes the frequencies."""

    dims: int
    base: float
    interleaved: bool = False
    scaling: BandScaling | YarnScaling | None = None

    def plain_frequencies(self) -> list[float]:
        return [self.base ** (-2 * i / self.dims) for i in range(self.dims // 2)]

    def frequencies(self) -> list[float]:
        return self.scaling.frequencies(self) if self.scaling is not None else self.plain_frequencies()

    @property
    def amplitude(self) -> float:
        return self.scaling.amplitude if self.scaling is not None else 1.0


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention over a shared per-token latent (see ``ops/latent.py``): low-rank queries, ``kv_rank`` cached latent
    channels plus one rotated key part for all heads, a causal sliding window, a softmax sink and a per-head gate."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int
    rot: RotarySpec

    type = "latent_attention"

    def __post_init__(self):
        assert self.rot.dims <= self.rot_dim and self.rot.dims % 2 == 0, "the rotation covers an even part of rot_dim"
        assert self.window >= 1

    @staticmethod
    def from_dict(m: dict) -> "LatentAttentionSpec":
        return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                   kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), scale=float(m["scale"]),
                                   window=int((m.get("mask") or {}).get("size") or NO_WINDOW),
                                   rot=RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"])))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
                "q_rank": self.q_rank, "scale": self.scale, "mask": {"size": self.window},
                "rot": {"dims": self.rot.dims, "base": self.rot.base}}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        H = self.heads
        return {p + "dq": (self.q_rank, width), p + "dq.norm": (self.q_rank,),
                p + "uq": (H * (self.dim + self.rot_dim), self.q_rank),
                p + "dkv": (self.kv_rank + self.rot_dim, width), p + "dkv.norm": (self.kv_rank,),
                p + "uk": (H * self.dim, self.kv_rank), p + "uv": (H * self.vdim, self.kv_rank),
                p + "sink": (H,), p + "g": (H, width), p + "o": (width, H * self.vdim)}


@dataclass(frozen=True)
class ClampedGluSpec:
    """``g sigmoid(1.702 g) (u + 1)`` with the gate capped at ``limit`` and the linear part clamped to ``+-limit``."""

    ff: int
    limit: float

    kind = "dense"

    @staticmethod
    def from_dict(m: dict) -> "ClampedGluSpec":
        return ClampedGluSpec(ff=int(m["ff"]), limit=float(m["limit"]))

    def to_dict(self) -> dict:
        return {"kind": self.kind, "ff": self.ff, "limit": self.limit}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        return {p + "gate": (self.ff, width), p + "up": (self.ff, width), p + "down": (width, self.ff)}


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention with a fixed decay per head (see ``ops/recurrent.py``): SiLU on queries, keys and values, one RMS norm
    over all heads, an element-wise output gate."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    type = "lightning"

    def __post_init__(self):
        assert len(self.decay) == self.heads, "one decay per head"

    @staticmethod
    def from_dict(m: dict) -> "LightningSpec":
        return LightningSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(x) for x in m["decay"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        n, nv = self.heads * self.dim, self.heads * self.vdim
        return {p + "q": (n, width), p + "k": (n, width), p + "v": (nv, width), p + "g": (nv, width), p + "norm": (nv,),
                p + "o": (width, nv)}


@dataclass(frozen=True)
class MatrixMemorySpec:
    """xLSTM matrix memory (see ``ops/recurrent.py``): exponential input gate and sigmoid forget gate per head with a running
    maximum, gate logits capped at ``gate_cap``, an RMS norm per head, an element-wise output gate."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float

    type = "mlstm"

    @staticmethod
    def from_dict(m: dict) -> "MatrixMemorySpec":
        return MatrixMemorySpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        H, n, nv = self.heads, self.heads * self.dim, self.heads * self.vdim
        return {p + "q": (n, width), p + "k": (n, width), p + "v": (nv, width), p + "g": (nv, width), p + "norm": (nv,),
                p + "o": (width, nv), p + "i": (H, width), p + "i.b": (H,), p + "f": (H, width), p + "f.b": (H,)}


@dataclass(frozen=True)
class QueryTemperature:
    """Queries at position ``p`` times ``1 + coef ln(floor((p + 1) / every) + 1)``."""

    coef: float
    every: int


@dataclass(frozen=True)
class KeyValueAttentionSpec:
    """Causal attention over grouped heads whose values are the projected keys (see ``ops/keyvalue.py``): one cached row per
    token and kv head, biases on the projections, a query temperature that grows with the position, a softmax sink and
    an element-wise output gate."""

    heads: int
    kv_heads: int
    dim: int
    scale: float
    q_temp: QueryTemperature

    type = "attention"

    def __post_init__(self):
        assert self.heads % self.kv_heads == 0, "query heads share kv heads evenly"

    @staticmethod
    def from_dict(m: dict) -> "KeyValueAttentionSpec":
        assert int(m.get("vdim", m["dim"])) == int(m["dim"]), "values are keys: vdim equals dim"
        t = m.get("q_temp") or {"coef": 0.0, "every": 1}
        return KeyValueAttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]),
                                     QueryTemperature(float(t["coef"]), int(t["every"])))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "scale": self.scale,
                "q_temp": {"coef": self.q_temp.coef, "every": self.q_temp.every}}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        n, nk = self.heads * self.dim, self.kv_heads * self.dim
        return {p + "q": (n, width), p + "q.b": (n,), p + "k": (nk, width), p + "k.b": (nk,), p + "sink": (self.heads,),
                p + "g": (n, width), p + "o": (width, n), p + "o.b": (width,)}


@dataclass(frozen=True)
class GluSpec:
    """``silu(gate) * up``."""

    ff: int

    kind = "dense"
    limit = None

    @staticmethod
    def from_dict(m: dict) -> "GluSpec":
        return GluSpec(ff=int(m["ff"]))

    def to_dict(self) -> dict:
        return {"kind": self.kind, "ff": self.ff}

    param_shapes = ClampedGluSpec.param_shapes


@dataclass(frozen=True)
class PolyNormSpec:
    """``a N(z) + b N(z^2) + c N(z^3) + e`` between two matrices, with the four numbers in a tensor and ``N`` the division by the root mean
    square over the ``ff`` values."""

    ff: int

    kind = "dense"

    @staticmethod
    def from_dict(m: dict) -> "PolyNormSpec":
        return PolyNormSpec(ff=int(m["ff"]))

    def to_dict(self) -> dict:
        return {"kind": self.kind, "ff": self.ff}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        return {p + "up": (self.ff, width), p + "down": (width, self.ff), p + "act": (4,)}


@dataclass(frozen=True)
class ExpertsRouting:
    """How a design weighs the chosen experts: ``scores`` is "softmax" or "sigmoid" of the router's logits; ``normalize``
    divides the chosen scores by their sum; the weight multiplies an expert's output, or its input with ``scale_input``."""

    scores: str = "softmax"
    normalize: bool = True
    scale_input: bool = False
    correction: bool = False           # the choice (not the weight) goes by score plus a constant per expert
    shared_gate: bool = False          # the shared unit's output times the sigmoid of one projected number


@dataclass(frozen=True)
class ExpertsSpec:
    """``experts`` gated units of which every token uses the ``top`` with the largest score, weighed as ``routing`` says;
    ``shared`` is a further unit that every token passes. ``identity`` more choices hand the input on as it is."""

    experts: int
    top: int
    expert: ClampedGluSpec | GluSpec
    routing: ExpertsRouting = ExpertsRouting()
    shared: GluSpec | None = None
    identity: int = 0

    kind = "moe"

    def __post_init__(self):
        assert 1 <= self.top <= self.choices
        assert not (self.identity and self.routing.scale_input), "a weight on an expert's input is no weight of an identity's output"

    @property
    def choices(self) -> int:
        return self.experts + self.identity

    @staticmethod
    def from_dict(m: dict, unit=ClampedGluSpec, routing: ExpertsRouting = ExpertsRouting()) -> "ExpertsSpec":
        shared = m.get("shared")
        return ExpertsSpec(int(m["router"]["experts"]), int(m["router"]["top"]), unit.from_dict(m["expert"]), routing,
                           unit.from_dict(shared) if shared else None, int(m["router"].get("identity") or 0))

    def to_dict(self) -> dict:
        def unit(u) -> dict:
            return {k: v for k, v in u.to_dict().items() if k != "kind"}

        d = {"kind": self.kind, "router": {"experts": self.experts, "top": self.top}, "expert": unit(self.expert)}
        if self.identity:
            d["router"]["identity"] = self.identity
        return {**d, "shared": unit(self.shared)} if self.shared is not None else d

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        out = {p + "router": (self.choices, width)}
        if self.routing.correction:
            out[p + "correction"] = (self.choices,)
        for e in range(self.experts):
            out.update(self.expert.param_shapes(f"{p}e{e}.", width))
        if self.shared is not None:
            out.update(self.shared.param_shapes(p + "shared.", width))
            if self.routing.shared_gate:
                out[p + "shared.sg"] = (1, width)
        return out


@dataclass(frozen=True)
class AttentionForm:
    """What a design fixes about a kind of grouped attention; sizes and constants are in ``GroupedAttentionSpec``.

    ``norm``: "projection" (RMS norm over all heads at once with weights, before the rotation), "head" (every head divided by its
    root mean square after the rotation) or "". ``span``: which keys ``j <= i`` a query sees, "all", "window" (``i - j < size``) or
    "chunk" (the same ``floor(position / size)``)."""

    type: str
    bias: bool = False
    conv: bool = False                 # a short causal convolution on every projected channel
    norm: str = ""
    interleaved: bool = False
    scaling: type | None = None        # BandScaling or YarnScaling
    span: str = "all"
    gate: bool = False                 # every head's output times the sigmoid of one projected number
    temperature: bool = False          # every head's scores times a number of its own

    def from_dict(self, m: dict) -> "GroupedAttentionSpec":
        rot, scaling = m["rot"], None
        if self.scaling is not None and rot.get("scaling"):
            scaling = self.scaling(**{k: float(v) for k, v in rot["scaling"].items()})
        return GroupedAttentionSpec(self, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                    RotarySpec(int(rot["dims"]), float(rot["base"]), self.interleaved, scaling),
                                    int(m["conv"]) if self.conv else 1, int(m["mask"]["size"]) if self.span != "all" else 0)


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Causal attention with grouped heads and cached keys and values (see ``ops/grouped.py``). ``taps`` of the convolution (1: the
    projection itself), ``size`` of the window or chunk."""

    form: AttentionForm
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    taps: int = 1
    size: int = 0

    def __post_init__(self):
        assert self.heads % self.kv_heads == 0, "query heads share kv heads evenly"
        assert self.rot.dims % 2 == 0 and self.rot.dims <= self.dim, "the rotation covers an even part of a head"
        assert self.taps >= 1 and (self.form.span == "all" or self.size >= 1)

    @property
    def type(self) -> str:
        return self.form.type

    @property
    def rows(self) -> tuple[int, int, int]:
        """Projected channels of queries, keys and values."""
        return self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim

    def to_dict(self) -> dict:
        rot = {"dims": self.rot.dims, "base": self.rot.base}
        if self.rot.scaling is not None:
            rot["scaling"] = asdict(self.rot.scaling)
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "rot": rot}
        if self.form.conv:
            d["conv"] = self.taps
        if self.form.span != "all":
            d["mask"] = {"size": self.size}
        return d

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        out: dict[str, tuple[int, ...]] = {}
        for name, n in zip("qkv", self.rows):
            out[p + name] = (n, width)
            if self.form.bias:
                out[p + name + ".b"] = (n,)
            if self.form.conv:
                out[p + name + ".conv"] = (n, self.taps)
            if self.form.norm == "projection" and name != "v":
                out[p + name + ".norm"] = (n,)
        if self.form.gate:
            out[p + "g"] = (self.heads, width)
        if self.form.temperature:
            out[p + "temp"] = (self.heads,)
        return {**out, p + "o": (width, self.heads * self.vdim)}


@dataclass(frozen=True)
class TimeMixSpec:
    """RWKV-style time mixing (see ``ops/recurrent.py``): projections of mixes with the previous token, a decay per key channel
    through a narrow product of ``decay_rank`` channels (0: as wide as the checkpoint's tensor), a bonus for the current token,
    an RMS norm per head, a SiLU gate."""

    heads: int
    dim: int
    decay_rank: int = 0

    type = "time_mix"
    DEFAULT_RANK = 32                  # of freshly initialised weights

    @staticmethod
    def from_dict(m: dict) -> "TimeMixSpec":
        return TimeMixSpec(int(m["heads"]), int(m["dim"]), int(m.get("decay_rank", 0)))

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim}
        return {**d, "decay_rank": self.decay_rank} if self.decay_rank else d

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        n, r = self.heads * self.dim, self.decay_rank or self.DEFAULT_RANK
        out = {f"{p}mu.{s}": (width,) for s in "rkvgw"}
        out.update({p + s: (n, width) for s in "rkvg"})
        return {**out, p + "w1": (r, width), p + "w2": (n, r), p + "w0": (n,), p + "u": (self.heads, self.dim), p + "norm": (n,), p + "o": (width, n)}

    def fitted(self, shapes: Callable[[str], tuple[int, ...]], p: str) -> "TimeMixSpec":
        rank = shapes(p + "w1")[0]
        assert self.decay_rank in (0, rank), f"{p}w1 has {rank} rows, the configuration says {self.decay_rank}"
        return replace(self, decay_rank=rank)


@dataclass(frozen=True)
class ForgetMixSpec:
    """Linear attention whose forget gate also decides what is written (HGRN2, see ``ops/recurrent.py``): a key row keeps ``f`` of itself
    and takes ``1 - f`` of the value, ``f`` between a lower bound per channel and 1; SiLU on the queries, an RMS norm per head with
    weights that the heads share."""

    heads: int
    dim: int
    vdim: int

    type = "forget_mix"

    @staticmethod
    def from_dict(m: dict) -> "ForgetMixSpec":
        return ForgetMixSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        n, nv = self.heads * self.dim, self.heads * self.vdim
        return {p + "q": (n, width), p + "f": (n, width), p + "f.b": (n,), p + "lower": (n,), p + "v": (nv, width), p + "norm": (self.vdim,),
                p + "o": (width, nv)}


@dataclass(frozen=True)
class DeltaRuleSpec:
    """Gated delta rule (see ``ops/recurrent.py``): short convolutions with SiLU on queries, keys and values, unit queries and keys that
    groups of heads share, a decay and a step size per head, an RMS norm per head with weights that the heads share, a SiLU gate."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    type = "delta"

    def __post_init__(self):
        assert self.heads % self.kv_heads == 0, "heads share queries and keys evenly"
        assert self.taps >= 1

    @staticmethod
    def from_dict(m: dict) -> "DeltaRuleSpec":
        return DeltaRuleSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.taps}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        H, n, nv = self.heads, self.kv_heads * self.dim, self.heads * self.vdim
        out: dict[str, tuple[int, ...]] = {}
        for name, rows in (("q", n), ("k", n), ("v", nv)):
            out[p + name], out[f"{p}{name}.conv"] = (rows, width), (rows, self.taps)
        return {**out, p + "b": (H, width), p + "a": (H, width), p + "A_log": (H,), p + "dt_bias": (H,), p + "g": (nv, width), p + "norm": (self.vdim,),
                p + "o": (width, nv)}


@dataclass(frozen=True)
class ParallelForm:
    """Which mixers a design puts side by side."""

    type: str
    left: AttentionForm
    right: type

    def from_dict(self, m: dict) -> "ParallelSpec":
        return ParallelSpec(self.type, self.left.from_dict(m["left"]), self.right.from_dict(m["right"]), float(m["left_scale"]), float(m["right_scale"]))


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same activations: ``left_scale * left + right_scale * right``."""

    type: str
    left: GroupedAttentionSpec
    right: TimeMixSpec
    left_scale: float
    right_scale: float

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        return {**self.left.param_shapes(p + "left.", width), **self.right.param_shapes(p + "right.", width)}

    def fitted(self, shapes: Callable[[str], tuple[int, ...]], p: str) -> "ParallelSpec":
        return replace(self, right=self.right.fitted(shapes, p + "right."))


@dataclass(frozen=True)
class NormedPairForm:
    """Which mixers a design puts side by side under norms of their own."""

    type: str
    left: AttentionForm
    right: type

    def from_dict(self, m: dict) -> "NormedPairSpec":
        return NormedPairSpec(self.type, self.left.from_dict(m["left"]), self.right.from_dict(m["right"]))


@dataclass(frozen=True)
class NormedPairSpec:
    """Two mixers that read the same activations: half the sum of their outputs, each RMS-normed over the width with a weight."""

    type: str
    left: GroupedAttentionSpec
    right: ForgetMixSpec

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        return {**self.left.param_shapes(p + "left.", width), **self.right.param_shapes(p + "right.", width), p + "left.out": (width,),
                p + "right.out": (width,)}


@dataclass(frozen=True)
class Design:
    """What all models of a design share. ``block`` is "post_norm" (sublayers read the stream; layer norm with bias and layer
    scale on their outputs), "parallel" (mixer and feed-forward read one RMS norm, and both are added) or "sandwich" (a norm before
    and after each sublayer: ``x += norm1b(mixer(norm1(x)))``, then ``x += norm2b(ff(norm2(x)))``)."""

    block: str
    tied: bool                         # the head is the embedding table
    mixers: dict                       # "type" in config.json -> what reads the layer's "mixer"
    feed_forwards: dict                # "kind" -> function that reads "mlp"
    unit_norms: bool = False           # norm weights are stored around zero
    bounded_norms: bool = False        # sandwich: norms are tanh(alpha x) * w + b (Dynamic Tanh) instead of RMS norms


WINDOW_ATTENTION = AttentionForm("window_attention", norm="projection", interleaved=True, span="window", gate=True)
TEMPERED_ATTENTION = AttentionForm("tempered_attention", bias=True, span="window", temperature=True)

DESIGNS = {
    "Lulezen": Design("post_norm", False, {"latent_attention": LatentAttentionSpec}, {"dense": ClampedGluSpec.from_dict}),
    "Zamusun": Design("parallel", True, {"lightning": LightningSpec, "mlstm": MatrixMemorySpec, "attention": KeyValueAttentionSpec},
                      {"dense": ClampedGluSpec.from_dict, "moe": ExpertsSpec.from_dict}, unit_norms=True),
    "Fogurax": Design("parallel", True,
                      {f.type: f for f in (AttentionForm("attention", bias=True, conv=True, norm="head", interleaved=True, scaling=BandScaling, gate=True),
                                           AttentionForm("attention_2", norm="projection", scaling=YarnScaling, span="chunk"),
                                           ParallelForm("parallel", WINDOW_ATTENTION, TimeMixSpec))},
                      {"dense": GluSpec.from_dict, "moe": partial(ExpertsSpec.from_dict, unit=GluSpec, routing=ExpertsRouting("sigmoid", False, True))}),
    "Sumitar": Design("sandwich", True, {"parallel": NormedPairForm("parallel", TEMPERED_ATTENTION, ForgetMixSpec), "delta": DeltaRuleSpec},
                      {"dense": PolyNormSpec.from_dict,
                       "moe": partial(ExpertsSpec.from_dict, unit=GluSpec, routing=ExpertsRouting(normalize=False, correction=True, shared_gate=True))},
                      bounded_norms=True),
}


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentAttentionSpec | LightningSpec | MatrixMemorySpec | KeyValueAttentionSpec | GroupedAttentionSpec | ParallelSpec | NormedPairSpec | DeltaRuleSpec
    mlp: ClampedGluSpec | GluSpec | PolyNormSpec | ExpertsSpec | None = None

    @staticmethod
    def from_dict(e: dict, design: Design) -> "LayerSpec":
        if e["type"] not in design.mixers:
            raise ValueError(f"unknown mixer {e['type']!r}; known: {sorted(design.mixers)}")
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] not in design.feed_forwards:
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: {sorted(design.feed_forwards)}")
        return LayerSpec(design.mixers[e["type"]].from_dict(e["mixer"]), design.feed_forwards[mlp["kind"]](mlp) if mlp is not None else None)

    def to_dict(self) -> dict:
        return {"type": self.mixer.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop-1`` run ``times`` times in a row with the same weights; each pass has its own cache and state
    and begins with ``x = W [x; embedding output]``."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class TokenSideSpec:
    """A second embedding of every token, ``dim`` channels for each layer, that enters the stream after the layer's sublayers:
    ``y = W_proj (gelu_tanh(W_gate x) * e)``, ``x += residual_mult * y / rms(y) * norm``."""

    dim: int


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer in a step."""

    layer: int
    enters: bool                       # a pass begins: the stream is mixed with the embedding output first


@dataclass(frozen=True)
class LayerStackConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float = 1e-6
    logit_softcap: float = 0.0         # 0: no cap
    eos_token_id: int = -1
    max_position_embeddings: int = 8192
    init_std: float = 0.02
    loop: LoopSpec | None = None
    residual_mult: float = 1.0         # factor of everything that is added to the stream
    token_side: TokenSideSpec | None = None

    # what the engine asks of every model configuration
    is_moe = False                     # (expert-parallel engines shard ModelConfig models only)

    def __post_init__(self):
        assert (self.residual_mult == 1.0 and self.token_side is None) or self.design.block == "parallel", "parallel blocks only"
        if self.loop is not None:
            assert 0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times >= 1, "loop range"

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def tie_word_embeddings(self) -> bool:
        return self.design.tied

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> tuple[LayerRun, ...]:
        """Layers in the order they run; a looped layer appears once per pass."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return tuple(LayerRun(i, False) for i in range(n))
        body = tuple(LayerRun(i, i == loop.start) for i in range(loop.start, loop.stop))
        return tuple(LayerRun(i, False) for i in range(loop.start)) + body * loop.times + tuple(LayerRun(i, False) for i in range(loop.stop, n))

    def param_shapes(self) -> dict[str, tuple[int, ...]]:
        d, post, sandwich = self.hidden_size, self.design.block == "post_norm", self.design.block == "sandwich"

        def norm(name: str) -> dict[str, tuple[int, ...]]:
            return {name: (d,), name + ".b": (d,), name + ".alpha": ()} if self.design.bounded_norms else {name: (d,)}

        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        if self.loop is not None:
            out["loop.in"] = (d, 2 * d)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            subs = [("1", "mix.", layer.mixer)] + ([("2", "mlp.", layer.mlp)] if layer.mlp is not None else [])
            for n, sub, spec in subs:
                if sandwich:
                    out.update({**norm(p + "norm" + n), **norm(p + "norm" + n + "b")})
                elif post:
                    out[p + "norm" + n] = out[p + "norm" + n + ".b"] = out[p + "ls" + n] = (d,)
                elif n == "1":
                    out[p + "norm1"] = (d,)
                out.update(spec.param_shapes(p + sub, d))
            if self.token_side is not None:
                out.update({p + "side.gate": (self.token_side.dim, d), p + "side.proj": (d, self.token_side.dim), p + "side.norm": (d,)})
        if self.token_side is not None:
            out["side.embed"] = (self.vocab_size, self.num_layers * self.token_side.dim)
        out.update(norm("final.norm"))
        if post:
            out["final.norm.b"] = (d,)
        if not self.design.tied:
            out["head"] = (self.vocab_size, d)
        return out

    def fill_value(self, name: str) -> float | None:
        """Constant a freshly initialised tensor starts from (None: random normal)."""
        last = name.rsplit(".", 1)[-1]
        if (last == "b" and not name.endswith(".mix.b")) or last in ("sink", "correction", "lower", "A_log"):
            return 0.0
        if last == "alpha":
            return 0.5
        if last in ("temp", "out"):
            return 1.0
        if last == "dt_bias":
            return -4.0
        if last == "act":
            return 1 / 3
        if last.startswith("norm") or last.startswith("ls"):
            return 0.0 if self.design.unit_norms and ".mix." not in name else 1.0
        if ".mu." in name or last == "conv":
            return 0.5
        return -3.0 if last == "w0" else None

    def fitted(self, weights: Mapping) -> "LayerStackConfig":
        """This configuration with the sizes that only the checkpoint's tensors tell."""
        def mixer(i: int, spec):
            return spec.fitted(lambda name: tuple(weights[name].shape), f"l{i}.mix.") if hasattr(spec, "fitted") else spec

        return replace(self, layers=tuple(replace(x, mixer=mixer(i, x.mixer)) for i, x in enumerate(self.layers)))

    def num_params(self) -> int:
        return sum(math.prod(s) for s in self.param_shapes().values())

    # ---- config.json -----------------------------------------------------------------------
    @staticmethod
    def from_dict(d: dict) -> "LayerStackConfig":
        loop, side = d.get("loop"), d.get("token_side")
        return LayerStackConfig(architecture=d["architecture"], vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                                layers=tuple(LayerSpec.from_dict(e, DESIGNS[d["architecture"]]) for e in d["layers"]), norm_eps=float(d["norm"]["eps"]),
                                logit_softcap=float(d.get("logit_softcap") or 0.0),
                                eos_token_id=int(d.get("eos_token_id", -1)),
                                loop=LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
                                residual_mult=float(d.get("residual_mult", 1.0)), token_side=TokenSideSpec(int(side["dim"])) if side else None)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [x.to_dict() for x in self.layers]}
        if self.logit_softcap > 0:
            d["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            d["loop"] = asdict(self.loop)
        if self.residual_mult != 1.0:
            d["residual_mult"] = self.residual_mult
        if self.token_side is not None:
            d["token_side"] = asdict(self.token_side)
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save(self, path: str | Path) -> None:
        Path(path).mkdir(parents=True, exist_ok=True)
        (Path(path) / "config.json").write_text(json.dumps(self.to_dict(), indent=2))

    def as_dict(self) -> dict:
        return asdict(self)


def uniform_stack(architecture: str, *, vocab: int, width: int, num_layers: int, mixer, mlp, **kw) -> LayerStackConfig:
    """A stack whose layers all have the same sizes."""
    return LayerStackConfig(architecture, vocab, width, (LayerSpec(mixer, mlp),) * num_layers, **kw)

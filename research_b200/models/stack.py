"""Configuration of models that are described layer by layer.

``ModelConfig`` holds one set of sizes for the whole model. A ``LayerStackConfig`` instead lists its layers; each names
the mixer it uses (with that layer's own sizes, window and rotation) and its feed-forward, or none. Mixers and
feed-forwards are small value types that know their ``config.json`` form and their tensors; a further kind is a new class
registered in ``MIXERS`` or ``FEED_FORWARDS``. How a layer is put together around them (norms, residual, head) is a
property of the design, a row of ``DESIGNS``.

``config.json`` form::

    {"architecture": "Lulezen", "vocab": V, "width": d, "norm": {"eps": e}, "logit_softcap": c,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", ...} or null}, ...]}

Tensors are named ``embed``, ``l<i>.norm1`` / ``.mix.*`` / ``.mlp.*``, ``final.norm``; matrices are stored ``[out, in]``.
Post-norm designs add ``.norm1.b`` / ``.ls1`` (and ``norm2`` / ``norm2.b`` / ``ls2`` for the feed-forward) and
``final.norm.b``; designs without tied embeddings have ``head``; looped stacks have ``loop.in``.
"""

from __future__ import annotations

import json
import math
from dataclasses import asdict, dataclass
from pathlib import Path


NO_WINDOW = 1 << 30          # a window nothing reaches: plain causal attention


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of pairs ``(i, i + dims/2)`` of the first ``dims`` channels by ``position * base^(-2i/dims)``."""

    dims: int
    base: float


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
class ExpertsSpec:
    """``experts`` clamped gated units of which every token uses the ``top`` with the largest softmax score, weighted by
    their scores divided by the chosen scores' sum."""

    experts: int
    top: int
    expert: ClampedGluSpec

    kind = "moe"

    def __post_init__(self):
        assert 1 <= self.top <= self.experts

    @staticmethod
    def from_dict(m: dict) -> "ExpertsSpec":
        return ExpertsSpec(int(m["router"]["experts"]), int(m["router"]["top"]), ClampedGluSpec.from_dict(m["expert"]))

    def to_dict(self) -> dict:
        return {"kind": self.kind, "router": {"experts": self.experts, "top": self.top},
                "expert": {"ff": self.expert.ff, "limit": self.expert.limit}}

    def param_shapes(self, p: str, width: int) -> dict[str, tuple[int, ...]]:
        out = {p + "router": (self.experts, width)}
        for e in range(self.experts):
            out.update(self.expert.param_shapes(f"{p}e{e}.", width))
        return out


MIXERS = {c.type: c for c in (LatentAttentionSpec, LightningSpec, MatrixMemorySpec, KeyValueAttentionSpec)}
FEED_FORWARDS = {c.kind: c for c in (ClampedGluSpec, ExpertsSpec)}


@dataclass(frozen=True)
class Design:
    """What all models of a design share. ``block`` is "post_norm" (sublayers read the stream; layer norm with bias and layer
    scale on their outputs) or "parallel" (mixer and feed-forward read one RMS norm whose weight is stored around zero, and
    both are added)."""

    block: str
    tied: bool                         # the head is the embedding table


DESIGNS = {"Lulezen": Design("post_norm", False), "Zamusun": Design("parallel", True)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentAttentionSpec | LightningSpec | MatrixMemorySpec | KeyValueAttentionSpec
    mlp: ClampedGluSpec | ExpertsSpec | None = None

    @staticmethod
    def from_dict(e: dict) -> "LayerSpec":
        if e["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {e['type']!r}; known: {sorted(MIXERS)}")
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] not in FEED_FORWARDS:
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: {sorted(FEED_FORWARDS)}")
        return LayerSpec(MIXERS[e["type"]].from_dict(e["mixer"]), FEED_FORWARDS[mlp["kind"]].from_dict(mlp) if mlp is not None else None)

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

    # what the engine asks of every model configuration
    is_moe = False                     # (expert-parallel engines shard ModelConfig models only)

    def __post_init__(self):
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
        d, post = self.hidden_size, self.design.block == "post_norm"
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        if self.loop is not None:
            out["loop.in"] = (d, 2 * d)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            subs = [("1", "mix.", layer.mixer)] + ([("2", "mlp.", layer.mlp)] if layer.mlp is not None else [])
            for n, sub, spec in subs:
                if post:
                    out[p + "norm" + n] = out[p + "norm" + n + ".b"] = out[p + "ls" + n] = (d,)
                elif n == "1":
                    out[p + "norm1"] = (d,)
                out.update(spec.param_shapes(p + sub, d))
        out["final.norm"] = (d,)
        if post:
            out["final.norm.b"] = (d,)
        if not self.design.tied:
            out["head"] = (self.vocab_size, d)
        return out

    def fill_value(self, name: str) -> float | None:
        """Constant a freshly initialised tensor starts from (None: random normal)."""
        last = name.rsplit(".", 1)[-1]
        if last == "b" or last == "sink":
            return 0.0
        if last.startswith("norm") or last.startswith("ls"):
            return 0.0 if self.design.block == "parallel" and ".mix." not in name else 1.0
        return None

    def num_params(self) -> int:
        return sum(math.prod(s) for s in self.param_shapes().values())

    # ---- config.json -----------------------------------------------------------------------
    @staticmethod
    def from_dict(d: dict) -> "LayerStackConfig":
        loop = d.get("loop")
        return LayerStackConfig(architecture=d["architecture"], vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                                layers=tuple(LayerSpec.from_dict(e) for e in d["layers"]), norm_eps=float(d["norm"]["eps"]),
                                logit_softcap=float(d.get("logit_softcap") or 0.0),
                                eos_token_id=int(d.get("eos_token_id", -1)),
                                loop=LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "layers": [x.to_dict() for x in self.layers]}
        if self.logit_softcap > 0:
            d["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            d["loop"] = asdict(self.loop)
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

"""Configuration of models that are described layer by layer.

``ModelConfig`` holds one set of sizes for the whole model. A ``LayerStackConfig`` instead lists its layers; each names
the mixer it uses (with that layer's own sizes, window and rotation) and its feed-forward, or none. Mixers and
feed-forwards are small value types that know their ``config.json`` form, their tensors and what they keep per token
in the paged cache; a further kind is a new class registered in ``MIXERS`` or ``FEED_FORWARDS``.

``config.json`` form::

    {"architecture": "Lulezen", "vocab": V, "width": d, "norm": {"eps": e}, "logit_softcap": c,
     "layers": [{"type": "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", ...} or null}, ...]}

Tensors are named ``embed``, ``l<i>.norm1`` / ``.norm1.b`` / ``.mix.*`` / ``.ls1`` (and ``norm2`` / ``mlp`` / ``ls2``
for the feed-forward), ``final.norm`` / ``final.norm.b`` and ``head``; matrices are stored ``[out, in]``.
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


MIXERS = {LatentAttentionSpec.type: LatentAttentionSpec}
FEED_FORWARDS = {ClampedGluSpec.kind: ClampedGluSpec}


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentAttentionSpec
    mlp: ClampedGluSpec | None = None

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

    # what the engine asks of every model configuration
    is_moe = False
    tie_word_embeddings = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def param_shapes(self) -> dict[str, tuple[int, ...]]:
        d = self.hidden_size
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            subs = [("1", "mix.", layer.mixer)] + ([("2", "mlp.", layer.mlp)] if layer.mlp is not None else [])
            for n, sub, spec in subs:
                out[p + "norm" + n] = out[p + "norm" + n + ".b"] = out[p + "ls" + n] = (d,)
                out.update(spec.param_shapes(p + sub, d))
        out["final.norm"] = out["final.norm.b"] = (d,)
        out["head"] = (self.vocab_size, d)
        return out

    @staticmethod
    def fill_value(name: str) -> float | None:
        """Constant a freshly initialised tensor starts from (None: random normal)."""
        last = name.rsplit(".", 1)[-1]
        if last == "b" or last == "sink":
            return 0.0
        if last.startswith("norm") or last.startswith("ls"):
            return 1.0
        return None

    def num_params(self) -> int:
        return sum(math.prod(s) for s in self.param_shapes().values())

    # ---- config.json -----------------------------------------------------------------------
    @staticmethod
    def from_dict(d: dict) -> "LayerStackConfig":
        return LayerStackConfig(architecture=d["architecture"], vocab_size=int(d["vocab"]), hidden_size=int(d["width"]),
                                layers=tuple(LayerSpec.from_dict(e) for e in d["layers"]), norm_eps=float(d["norm"]["eps"]),
                                logit_softcap=float(d.get("logit_softcap") or 0.0),
                                eos_token_id=int(d.get("eos_token_id", -1)))

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.norm_eps}, "logit_softcap": self.logit_softcap, "layers": [x.to_dict() for x in self.layers]}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save(self, path: str | Path) -> None:
        Path(path).mkdir(parents=True, exist_ok=True)
        (Path(path) / "config.json").write_text(json.dumps(self.to_dict(), indent=2))

    def as_dict(self) -> dict:
        return asdict(self)


def uniform_stack(architecture: str, *, vocab: int, width: int, num_layers: int, mixer: LatentAttentionSpec,
                  mlp: ClampedGluSpec | None, **kw) -> LayerStackConfig:
    """A stack whose layers all have the same sizes."""
    return LayerStackConfig(architecture, vocab, width, (LayerSpec(mixer, mlp),) * num_layers, **kw)

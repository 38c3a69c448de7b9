"""Two mixers side by side as parts of a layer stack.

``ParallelPart``: attention (``grouped.py``) and time mixing (``recurrent.py``) read the same activations, write next to each other and
share one output projection. The factor of each half is applied in fp32 before that: in the head gate on the left, in the norm's
weight on the right.

``NormedPairPart``: attention and forget mixing share one joint projection, and each has its own output projection, since every half is
normed over the width before they are added (by whoever adds them to the stream)."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ... import ops
from ...models.stack import NormedPairSpec, ParallelSpec
from .base import Part
from .grouped import GroupedPart, GroupedWeights
from .recurrent import ForgetMixPart, ForgetMixWeights, TimeMixPart, TimeMixWeights


@dataclass
class ParallelWeights:
    spec: ParallelSpec
    left: GroupedWeights
    right: TimeMixWeights
    wo: torch.Tensor             # [wp, left heads | right heads]

    @property
    def wproj(self) -> torch.Tensor:         # (whose last rows are the layer's narrow projection)
        return self.left.wproj

    @property
    def left_columns(self) -> int:
        return self.left.geo.heads * self.left.geo.dp


class ParallelPart(Part):
    fuses_tail = True

    def __init__(self, runner):
        super().__init__(runner)
        self.left, self.right = runner._part(GroupedPart), runner._part(TimeMixPart)

    @staticmethod
    def cache_row_elements(spec) -> int:
        return GroupedPart.cache_row_elements(spec.left)

    @staticmethod
    def state_floats(spec) -> int:
        return GroupedPart.state_floats(spec.left) + TimeMixPart.state_floats(spec.right)

    @staticmethod
    def small_rows(spec) -> int:
        return GroupedPart.small_rows(spec.left)

    def make(self, spec: ParallelSpec, tail: int = 0) -> ParallelWeights:
        left, right = self.left.make(spec.left, tail, output=False), self.right.make(spec.right, output=False)
        w = ParallelWeights(spec, left, right, self.zeros(self.r.wp, left.geo.heads * left.geo.dp + right.geo.heads * right.geo.vp))
        self.layers.append(w)
        return w

    def new_cache(self, w: ParallelWeights):
        return self.left.new_cache(w.left), self.right.new_cache(w.right)

    def allocate(self) -> None:
        self.out = self.zeros(self.r.rows * max(w.wo.shape[1] for w in self.layers))

    def load(self, w: ParallelWeights, get, p: str) -> None:
        self.left.load(w.left, get, p + "left.")
        self.right.load(w.right, get, p + "right.", w.spec.right_scale)
        self.left.load_output(w.left, get, p + "left.", w.wo[:, :w.left_columns])
        self.right.load_output(w.right, get, p + "right.", w.wo[:, w.left_columns:])

    def load_small(self, w: ParallelWeights, get, p: str, dst: torch.Tensor) -> None:
        self.left.load_small(w.left, get, p + "left.", dst)

    def plan(self, b):
        return self.left.planned(b), self.right.planned(b)

    def project(self, w: ParallelWeights, inp, tail) -> None:
        self.left.project(w.left, inp, tail)

    def forward(self, w: ParallelWeights, cache, inp, y, b, plan, small=None) -> None:
        T, n = b.num_tokens, w.left_columns
        out = self.out[:T * w.wo.shape[1]].view(T, -1)
        self.left.attend(w.left, cache[0], out[:, :n], b, plan[0], small, w.spec.left_scale)
        self.right.mix(w.right, cache[1], inp, out[:, n:], b, plan[1])
        ops.gemm(out, w.wo, out=y, out_f32=True)


@dataclass
class NormedPairWeights:
    spec: NormedPairSpec
    left: GroupedWeights
    right: ForgetMixWeights
    wproj: torch.Tensor          # right queries | right values | left | logits of the right's forget gate
    bproj: torch.Tensor | None
    left_out: torch.Tensor       # [wp] weights of the halves' norms
    right_out: torch.Tensor


class NormedPairPart(Part):
    fuses_tail = True

    def __init__(self, runner):
        super().__init__(runner)
        if not runner.sandwich:
            raise ValueError("two mixers under norms of their own belong to sandwich blocks")
        self.left, self.right = runner._part(GroupedPart), runner._part(ForgetMixPart)

    @staticmethod
    def cache_row_elements(spec) -> int:
        return GroupedPart.cache_row_elements(spec.left)

    @staticmethod
    def state_floats(spec) -> int:
        return GroupedPart.state_floats(spec.left) + ForgetMixPart.state_floats(spec.right)

    @staticmethod
    def small_rows(spec) -> int:
        return ForgetMixPart.geometry(spec.right).offsets[1]

    def make(self, spec: NormedPairSpec, tail: int = 0) -> NormedPairWeights:
        assert not spec.left.form.gate, "the narrow projection holds the forget gate's logits alone"
        left, right = self.left.make(spec.left, projection=False), self.right.make(spec.right)
        n, m = right.geo.proj, left.geo.proj
        w = NormedPairWeights(spec, left, right, self.zeros(n + m + tail, self.r.wp), self.zeros(n + m + tail) if spec.left.form.bias else None,
                              *(self.zeros(self.r.wp, dtype=torch.float32) for _ in range(2)))
        right.wproj, left.wproj = w.wproj[:n], w.wproj[n:n + m]
        left.bproj = w.bproj[n:n + m] if w.bproj is not None else None
        self.layers.append(w)
        return w

    def new_cache(self, w: NormedPairWeights):
        return self.left.new_cache(w.left), self.right.new_cache(w.right)

    def allocate(self) -> None:
        self.proj = self.zeros(self.r.rows * max(w.right.geo.proj + w.left.geo.proj for w in self.layers))

    def load(self, w: NormedPairWeights, get, p: str) -> None:
        self.left.load(w.left, get, p + "left.")
        self.right.load(w.right, get, p + "right.")
        for dst, name in ((w.left_out, "left.out"), (w.right_out, "right.out")):
            dst[:self.r.cfg.hidden_size].copy_(get(p + name).float())

    def load_small(self, w: NormedPairWeights, get, p: str, dst: torch.Tensor) -> None:
        self.right.load_small(w.right, get, p + "right.", dst)

    def plan(self, b):
        return self.left.planned(b), self.right.planned(b)

    def _projected(self, w: NormedPairWeights, T: int) -> torch.Tensor:
        n = w.right.geo.proj + w.left.geo.proj
        return self.proj[:T * n].view(T, n)

    def project(self, w: NormedPairWeights, inp, tail) -> None:
        ops.gemm(inp, w.wproj, bias=w.bproj, out=self._projected(w, inp.shape[0]), silu_cols=w.right.geo.silu_cols, tail=tail)

    def forward(self, w: NormedPairWeights, cache, inp, y, b, plan, small=None) -> dict:
        T, n = b.num_tokens, w.left.geo.heads * w.left.geo.dp
        proj = self._projected(w, T)
        out = self.left.out[:T * n].view(T, n)
        self.left.attend(w.left, cache[0], out, b, plan[0], None, proj=proj[:, w.right.geo.proj:])
        ops.gemm(out, w.left.wo, out=y, out_f32=True)
        other = self.r.y2[:T]
        self.right.mix(w.right, cache[1], proj, small, other, b, plan[1])
        return {"y1": y, "pair": (other, w.left_out, w.right_out)}

"""Two mixers side by side as a part of a layer stack: attention (``grouped.py``) and time mixing (``recurrent.py``) read the same
activations, write next to each other and share one output projection. The factor of each half is applied in fp32 before that:
in the head gate on the left, in the norm's weight on the right."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ... import ops
from ...models.stack import ParallelSpec
from .base import Part
from .grouped import GroupedPart, GroupedWeights
from .recurrent import TimeMixPart, TimeMixWeights


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

"""Feed-forwards as parts of a layer stack: a gated unit, clamped or plain SiLU, dense (gate|up with the unit in the GEMM's epilogue,
down) or as routed experts (``ops/experts.py``) with or without a shared one."""

from __future__ import annotations

import torch

from ... import ops
from ...models.stack import ClampedGluSpec, ExpertsSpec, GluSpec
from ...ops.experts import ExpertsGeometry, ExpertsScratch
from .base import Part, up

GLU_BN = 256                                    # tile width of the fused gate|up launch


class DenseWeights:
    __slots__ = ("spec", "wgu", "wd", "ffp")


class DensePart(Part):
    def make(self, spec: ClampedGluSpec | GluSpec) -> DenseWeights:
        r = self.r
        w = DenseWeights()
        w.spec = spec
        w.ffp = up(spec.ff, GLU_BN // 2 if r.bf16 else 8)
        w.wgu, w.wd = self.zeros(2 * w.ffp, r.wp), self.zeros(r.wp, w.ffp)
        self.layers.append(w)
        return w

    def allocate(self) -> None:
        most = self.r.rows * max(w.ffp for w in self.layers)
        self.act = self.zeros(most)
        self.gu = None if self.r.bf16 else self.zeros(2 * most)

    def load(self, w: DenseWeights, get, p: str) -> None:
        gate, upw = get(p + "gate"), get(p + "up")
        ff, d = w.spec.ff, self.r.cfg.hidden_size
        if self.r.bf16:        # interleaved blocks for the fused epilogue; padding rows give 0
            pad = self.zeros(2, w.ffp, self.r.wp)
            pad[0, :ff, :d], pad[1, :ff, :d] = gate, upw
            w.wgu.copy_(ops.interleave_gate_up(pad[0], pad[1], GLU_BN))
        else:
            w.wgu[:ff, :d].copy_(gate)
            w.wgu[w.ffp:w.ffp + ff, :d].copy_(upw)
        w.wd[:d, :ff].copy_(get(p + "down"))

    def forward(self, w: DenseWeights, inp, y, small=None) -> dict:
        """Addends of the residual stream (arguments of ``ops.stream_norm``)."""
        T = inp.shape[0]
        act = self.act[:T * w.ffp].view(T, w.ffp)
        if self.r.bf16:
            ops.gemm(inp, w.wgu, out=act, bn=GLU_BN, swiglu=True, glu_limit=w.spec.limit)
        else:
            gu = ops.gemm(inp, w.wgu, out=self.gu[:T * 2 * w.ffp].view(T, 2 * w.ffp))
            ops.clamped_glu(gu, w.spec.limit, out=act)
        ops.gemm(act, w.wd, out=y, out_f32=True)
        return {"y2": y}


class ExpertsWeights:
    __slots__ = ("spec", "geo", "wgu", "wd", "shared")


class ExpertsPart(Part):
    @staticmethod
    def small_rows(spec: ExpertsSpec) -> int:
        return spec.experts

    def make(self, spec: ExpertsSpec) -> ExpertsWeights:
        r = self.r
        w = ExpertsWeights()
        w.spec = spec
        how = spec.routing
        w.geo = ExpertsGeometry.make(spec.experts, spec.top, spec.expert.ff, r.wp, spec.expert.limit, r.dtype, how.scores, how.normalize, how.scale_input)
        w.shared = r._part(DensePart).make(spec.shared) if spec.shared is not None else None
        w.wgu, w.wd = self.zeros(spec.experts * 2 * w.geo.ffp, r.wp), self.zeros(spec.experts * r.wp, w.geo.ffp)
        self.layers.append(w)
        return w

    def allocate(self) -> None:
        self.scratch = {g: ExpertsScratch(g, self.r.rows, self.r.dtype, self.r.device) for g in {w.geo for w in self.layers}}

    def load(self, w: ExpertsWeights, get, p: str) -> None:
        n = range(w.spec.experts)
        ops.pack_experts((get(f"{p}e{e}.gate") for e in n), (get(f"{p}e{e}.up") for e in n), (get(f"{p}e{e}.down") for e in n), w.geo, w.wgu, w.wd)
        if w.shared is not None:
            self.r._part(DensePart).load(w.shared, get, p + "shared.")

    def load_small(self, w: ExpertsWeights, get, p: str, dst: torch.Tensor) -> None:
        dst[:w.spec.experts, :self.r.cfg.hidden_size].copy_(get(p + "router"))

    def forward(self, w: ExpertsWeights, inp, y, small) -> dict:
        e, p = ops.experts_forward(inp, small, w.geo, self.scratch[w.geo], w.wgu, w.wd)
        add = {"experts": e, "expert_weights": p, "top": w.geo.top}
        return {**self.r._part(DensePart).forward(w.shared, inp, y), **add} if w.shared is not None else add

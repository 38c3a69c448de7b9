"""Feed-forwards as parts of a layer stack: a gated unit, clamped or plain SiLU, dense (gate|up with the unit in the GEMM's epilogue,
down) or as routed experts (``ops/experts.py``) with or without a shared one; two matrices with normed powers between them."""

from __future__ import annotations

import torch

from ... import ops
from ...models.stack import ClampedGluSpec, ExpertsSpec, GluSpec, PolyNormSpec
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


class PolyNormWeights:
    __slots__ = ("spec", "wu", "wd", "act", "ffp")


class PolyNormPart(Part):
    def make(self, spec: PolyNormSpec) -> PolyNormWeights:
        w = PolyNormWeights()
        w.spec, w.ffp = spec, up(spec.ff, 8)
        w.wu, w.wd = self.zeros(w.ffp, self.r.wp), self.zeros(self.r.wp, w.ffp)
        w.act = self.zeros(4, dtype=torch.float32)
        self.layers.append(w)
        return w

    def allocate(self) -> None:
        self.z, self.a = (self.zeros(self.r.rows * max(w.ffp for w in self.layers)) for _ in range(2))

    def load(self, w: PolyNormWeights, get, p: str) -> None:
        ff, d = w.spec.ff, self.r.cfg.hidden_size
        w.wu[:ff, :d].copy_(get(p + "up"))
        w.wd[:d, :ff].copy_(get(p + "down"))
        w.act.copy_(get(p + "act").float())

    def forward(self, w: PolyNormWeights, inp, y, small=None) -> dict:
        T = inp.shape[0]
        z, a = (t[:T * w.ffp].view(T, w.ffp) for t in (self.z, self.a))
        ops.gemm(inp, w.wu, out=z)
        ops.poly_norm(z, w.act, w.spec.ff, self.r.cfg.norm_eps, a)
        ops.gemm(a, w.wd, out=y, out_f32=True)
        return {"y2": y}


class ExpertsWeights:
    __slots__ = ("spec", "geo", "wgu", "wd", "shared", "correction")


class ExpertsPart(Part):
    @staticmethod
    def small_rows(spec: ExpertsSpec) -> int:
        return spec.choices + int(spec.routing.shared_gate and spec.shared is not None)

    def make(self, spec: ExpertsSpec) -> ExpertsWeights:
        r = self.r
        w = ExpertsWeights()
        w.spec = spec
        how = spec.routing
        w.geo = ExpertsGeometry.make(spec.experts, spec.top, spec.expert.ff, r.wp, spec.expert.limit, r.dtype, how.scores, how.normalize, how.scale_input, spec.identity)
        w.correction = self.zeros(spec.choices, dtype=torch.float32) if how.correction else None
        w.shared = r._part(DensePart).make(spec.shared) if spec.shared is not None else None
        w.wgu, w.wd = self.zeros(spec.experts * 2 * w.geo.ffp, r.wp), self.zeros(spec.experts * r.wp, w.geo.ffp)
        self.layers.append(w)
        return w

    def allocate(self) -> None:
        self.scratch = {g: ExpertsScratch(g, self.r.rows, self.r.dtype, self.r.device) for g in {w.geo for w in self.layers}}

    def load(self, w: ExpertsWeights, get, p: str) -> None:
        n = range(w.spec.experts)
        ops.pack_experts((get(f"{p}e{e}.gate") for e in n), (get(f"{p}e{e}.up") for e in n), (get(f"{p}e{e}.down") for e in n), w.geo, w.wgu, w.wd)
        if w.correction is not None:
            w.correction.copy_(get(p + "correction").float())
        if w.shared is not None:
            self.r._part(DensePart).load(w.shared, get, p + "shared.")

    def load_small(self, w: ExpertsWeights, get, p: str, dst: torch.Tensor) -> None:
        n, d = w.spec.choices, self.r.cfg.hidden_size
        dst[:n, :d].copy_(get(p + "router"))
        if self.small_rows(w.spec) > n:
            dst[n:n + 1, :d].copy_(get(p + "shared.sg"))

    def forward(self, w: ExpertsWeights, inp, y, small) -> dict:
        sc = self.scratch[w.geo]
        e, p = ops.experts_forward(inp, small, w.geo, sc, w.wgu, w.wd, w.correction)
        if self.r.sandwich:
            add = {"chosen": ops.ChosenExperts(e, p, sc.idx[:inp.shape[0]], w.geo.experts, inp)}
            if w.shared is not None and w.spec.routing.shared_gate:
                add["gate"] = small[:, w.spec.choices:]
        else:
            add = {"experts": e, "expert_weights": p, "top": w.geo.top}
        return {**self.r._part(DensePart).forward(w.shared, inp, y), **add} if w.shared is not None else add

"""Recurrent mixers (``ops/recurrent.py``) as a part of a layer stack: one joint projection (queries, keys, values, output
gate), the recurrence over the sequences' state slots, one norm-and-gate kernel, the output projection. Gate logits of the
recurrence come from the layer's narrow fp32 projection. Decoded tokens and portions of at most ``SCAN_PORTION`` tokens run
token by token, longer ones in chunks on the tensor cores, in one batch."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ... import ops
from ...models.stack import DeltaRuleSpec, ForgetMixSpec, LightningSpec, MatrixMemorySpec, TimeMixSpec
from ...ops.recurrent import (MAX_DIM, MAX_TAPS, ChunkTable, DeltaRule, ForgetMix, RecurrentGeometry, RecurrentState, TimeMix, chunk_workspace,
                              chunked_supported, delta_chunked_supported, delta_workspace, time_mix_chunked_supported, time_mix_workspace)
from .base import Part, load_head_columns, load_head_vector, load_heads, up

SCAN_PORTION = 16            # new tokens of a sequence up to which the recurrence runs token by token


def recurrent_geometry(m: LightningSpec | MatrixMemorySpec) -> RecurrentGeometry:
    gated = isinstance(m, MatrixMemorySpec)
    return RecurrentGeometry(m.heads, m.dim, m.vdim, silu=not gated, gated=gated)


class RecurrentWeights:
    __slots__ = ("geo", "spec", "wproj", "wo", "norm", "decay", "bias_i", "bias_f", "cap")


class RecurrentPart(Part):
    fuses_tail = True

    @staticmethod
    def state_floats(spec) -> int:
        return recurrent_geometry(spec).state_floats

    @staticmethod
    def small_rows(spec) -> int:
        return 2 * spec.heads if isinstance(spec, MatrixMemorySpec) else 0

    def make(self, spec, tail: int = 0) -> RecurrentWeights:
        g, f32 = recurrent_geometry(spec), torch.float32
        if g.kp > MAX_DIM:
            raise ValueError(f"the recurrent kernels take up to {MAX_DIM} key channels per head")
        w = RecurrentWeights()
        w.spec, w.geo = spec, g
        w.wproj, w.wo = self.zeros(g.proj + tail, self.r.wp), self.zeros(self.r.wp, g.heads * g.vp)
        w.norm = self.zeros(g.heads * g.vp, dtype=f32)
        w.decay = w.bias_i = w.bias_f = None
        w.cap = 1.0
        if g.gated:
            w.bias_i, w.bias_f, w.cap = self.zeros(g.heads, dtype=f32), self.zeros(g.heads, dtype=f32), spec.gate_cap
        else:
            w.decay = torch.tensor(spec.decay, dtype=f32, device=self.r.device)
        self.layers.append(w)
        return w

    def new_cache(self, w) -> RecurrentState:
        return RecurrentState.zeros(w.geo, self.r.scratch_state_slot + 1, self.r.device)

    def allocate(self) -> None:
        r = self.r
        self.proj = self.zeros(r.rows * max(w.geo.proj for w in self.layers))
        most = r.rows * max(w.geo.heads * w.geo.vp for w in self.layers)
        self.o = self.zeros(most, dtype=torch.float32)
        self.out = self.zeros(most)

    def load(self, w: RecurrentWeights, get, p: str) -> None:
        g = w.geo
        H, (_, ok, ov, og) = g.heads, g.offsets
        load_heads(w.wproj[:ok], get(p + "q"), H, g.dim, g.kp)
        load_heads(w.wproj[ok:ov], get(p + "k"), H, g.dim, g.kp)
        load_heads(w.wproj[ov:og], get(p + "v"), H, g.vdim, g.vp)
        load_heads(w.wproj[og:g.proj], get(p + "g"), H, g.vdim, g.vp)
        load_head_columns(w.wo, get(p + "o"), H, g.vdim, g.vp)
        load_head_vector(w.norm, get(p + "norm").float(), H, g.vdim, g.vp)
        if g.gated:
            w.bias_i.copy_(get(p + "i.b").float())
            w.bias_f.copy_(get(p + "f.b").float())

    def load_small(self, w: RecurrentWeights, get, p: str, dst: torch.Tensor) -> None:
        if w.geo.gated:
            dst[:w.geo.heads, :self.r.cfg.hidden_size].copy_(get(p + "i"))
            dst[w.geo.heads:2 * w.geo.heads, :self.r.cfg.hidden_size].copy_(get(p + "f"))

    def _projected(self, w: RecurrentWeights, T: int) -> torch.Tensor:
        return self.proj[:T * w.geo.proj].view(T, w.geo.proj)

    def project(self, w: RecurrentWeights, inp, tail) -> None:
        ops.gemm(inp, w.wproj, out=self._projected(w, inp.shape[0]), silu_cols=w.geo.silu_cols, tail=tail)

    def forward(self, w: RecurrentWeights, state: RecurrentState, inp, y, b, plan, small=None) -> None:
        T, g = b.num_tokens, w.geo
        n = g.heads * g.vp
        proj = self._projected(w, T)
        o, out = self.o[:T * n].view(T, n), self.out[:T * n].view(T, n)
        self.recur(w, state, proj, small, o, b, plan)
        ops.gated_norm(o, w.norm, proj[:, g.offsets[3]:], g, self.r.cfg.norm_eps, out, g.gated)
        ops.gemm(out, w.wo, out=y, out_f32=True)

    def plan(self, b):
        """(sequences and rows that run token by token, chunk table of the rest)"""
        if b.cu_q is None or not self.r.bf16:
            return b.rows, b.num_tokens, None
        first = next((i for i in range(b.rows) if b.host_cu_q[i + 1] - b.host_cu_q[i] > SCAN_PORTION), b.rows)
        return first, b.host_cu_q[first], ChunkTable.make(b.host_cu_q, first, self.r.device) if first < b.rows else None

    def recur(self, w: RecurrentWeights, state: RecurrentState, proj, small, o, b, plan) -> None:
        """``o`` from the projected rows, and the state of the batch's sequences moved on."""
        g = w.geo
        n_seq, rows, table = plan
        if table is not None and not chunked_supported(g):
            n_seq, rows, table = b.rows, b.num_tokens, None
        args = (proj, small, g, w.decay, w.bias_i, w.bias_f, w.cap, state, b.state_slots)
        if b.n_single > 0:
            ops.recurrent_scan(*args, None, b.seq_lens, o, b.n_single, b.n_single)
        if n_seq > b.n_single:
            ops.recurrent_scan(*args, b.cu_q, b.seq_lens, o, rows, n_seq, b.n_single)
        if table is not None:
            room = torch.empty(chunk_workspace(table.chunks.shape[0], g), dtype=torch.uint8, device=o.device)
            ops.recurrent_chunks(*args, b.cu_q, b.seq_lens, o, table, room)


MIXES = "rkvgw"              # what reads a mix of its own: the joint projection's four parts and the decay
WIDE_BATCH = 512             # rows from which the four projections are products of their own


class TimeMixWeights:
    __slots__ = ("geo", "spec", "wproj", "w1", "w2", "w0", "bonus", "mu", "norm", "wo", "rank")


@dataclass
class TimeMixState:
    state: RecurrentState
    history: torch.Tensor        # [slots, 1, wp], the last input of every sequence


class TimeMixPart(Part):
    @staticmethod
    def geometry(spec: TimeMixSpec) -> RecurrentGeometry:
        return RecurrentGeometry(spec.heads, spec.dim, spec.dim, silu=False, gated=False)

    @staticmethod
    def state_floats(spec) -> int:
        return TimeMixPart.geometry(spec).state_floats

    def make(self, spec: TimeMixSpec, tail: int = 0, output: bool = True) -> TimeMixWeights:
        g, r, f32 = self.geometry(spec), self.r, torch.float32
        if g.kp > MAX_DIM:
            raise ValueError(f"the recurrent kernels take up to {MAX_DIM} key channels per head")
        w = TimeMixWeights()
        w.spec, w.geo, w.rank = spec, g, up(spec.decay_rank, 8)
        n = g.heads * g.kp
        w.wproj = self.zeros(4 * n, r.wp)
        w.w1, w.w2 = self.zeros(w.rank, r.wp), self.zeros(n, w.rank * self.parts)
        w.w0, w.bonus, w.norm = (self.zeros(n, dtype=f32) for _ in range(3))
        w.mu = self.zeros(len(MIXES), r.wp, dtype=f32)
        w.wo = self.zeros(r.wp, n) if output else None
        self.layers.append(w)
        return w

    @property
    def parts(self) -> int:      # how many activations carry one value of the decay's inner product exactly enough
        return 1 if self.r.dtype == torch.float32 else 2

    def new_cache(self, w: TimeMixWeights) -> TimeMixState:
        slots = self.r.scratch_state_slot + 1
        return TimeMixState(RecurrentState.zeros(w.geo, slots, self.r.device), self.zeros(slots, 1, self.r.wp))

    def allocate(self) -> None:
        r, f32 = self.r, torch.float32
        n, rank = max(w.geo.heads * w.geo.kp for w in self.layers), max(w.rank for w in self.layers)
        self.mixed = self.zeros(len(MIXES), r.rows, r.wp)
        self.proj = self.zeros(r.rows * 4 * n)
        self.inner, self.tanh = self.zeros(r.rows * rank, dtype=f32), self.zeros(r.rows * rank * self.parts)
        self.z, self.o = self.zeros(r.rows * n, dtype=f32), self.zeros(r.rows * n, dtype=f32)
        self.out = self.zeros(r.rows * max([w.geo.heads * w.geo.vp for w in self.layers if w.wo is not None], default=0))

    def load(self, w: TimeMixWeights, get, p: str, factor: float = 1.0) -> None:
        """``factor`` of the output, carried by the norm's weight."""
        g, d = w.geo, self.r.cfg.hidden_size
        for i, s in enumerate(MIXES):
            w.mu[i, :d].copy_(get(f"{p}mu.{s}").float())
            if s != "w":
                load_heads(w.wproj[i * g.heads * g.kp:(i + 1) * g.heads * g.kp], get(p + s), g.heads, g.dim, g.kp)
        rank = w.spec.decay_rank
        w.w1[:rank, :d].copy_(get(p + "w1"))
        for i in range(self.parts):
            load_heads(w.w2[:, i * w.rank:], get(p + "w2"), g.heads, g.dim, g.kp)
        load_head_vector(w.w0, get(p + "w0").float(), g.heads, g.dim, g.kp)
        load_head_vector(w.bonus, get(p + "u").float().reshape(-1), g.heads, g.dim, g.kp)
        load_head_vector(w.norm, get(p + "norm").float() * factor, g.heads, g.vdim, g.vp)
        if w.wo is not None:
            self.load_output(w, get, p, w.wo)

    def load_output(self, w: TimeMixWeights, get, p: str, dst: torch.Tensor) -> None:
        load_head_columns(dst, get(p + "o"), w.geo.heads, w.geo.vdim, w.geo.vp)

    plan = RecurrentPart.plan

    def mix(self, w: TimeMixWeights, cache: TimeMixState, inp, out, b, plan) -> None:
        """Normed and gated heads' outputs into ``out [T, H * vp]``."""
        T = b.num_tokens
        ops.token_shift(inp, w.mu, self.mixed, cache.history, b.cu_q, b.positions, b.state_slots)
        self.recur(w, cache, self.project_mixes(w, T), self.decay_logits(w, T), out, b, plan)

    def project_mixes(self, w: TimeMixWeights, T: int) -> torch.Tensor:
        """``r | k | v | gate`` of the mixes."""
        n = w.geo.heads * w.geo.kp
        proj = self.proj[:self.r.rows * 4 * n].view(-1, 4 * n)
        if T < WIDE_BATCH:
            ops.head_gemm_expand(self.mixed[:4], w.wproj, proj, T)       # (the whole buffer: its destination table is kept)
            return proj[:T]
        for i in range(4):
            ops.gemm(self.mixed[i, :T], w.wproj[i * n:(i + 1) * n], out=proj[:T, i * n:(i + 1) * n])
        return proj[:T]

    def decay_logits(self, w: TimeMixWeights, T: int) -> torch.Tensor:
        """``W_w2 tanh(W_w1 mix)`` in fp32."""
        n = w.geo.heads * w.geo.kp
        inner, tanh = self.inner[:T * w.rank].view(T, -1), self.tanh[:T * w.rank * self.parts].view(T, -1)
        ops.gemm(self.mixed[4, :T], w.w1, out=inner, out_f32=True)
        ops.tanh_parts(inner, tanh)
        return ops.gemm(tanh, w.w2, out=self.z[:T * n].view(T, n), out_f32=True)

    def recur(self, w: TimeMixWeights, cache: TimeMixState, proj, z, out, b, plan) -> None:
        T, g, eps = b.num_tokens, w.geo, self.r.cfg.norm_eps
        mix = TimeMix(z, w.w0, w.bonus)
        n_seq, rows, table = plan if time_mix_chunked_supported(g) else (b.rows, T, None)
        single = b.rows if b.cu_q is None else b.n_single
        if single > 0:
            ops.time_mix_decode(proj, g, mix, cache.state, b.state_slots, b.seq_lens, w.norm, eps, out, single)
        if n_seq > single:
            o = self.o[:T * g.heads * g.vp].view(T, -1)
            ops.recurrent_scan(proj, None, g, None, None, None, 1.0, cache.state, b.state_slots, b.cu_q, b.seq_lens, o, rows, n_seq, single, mix=mix)
            ops.gated_norm(o[single:rows], w.norm, proj[single:, g.offsets[3]:], g, eps, out[single:], True, silu=True)
        if table is not None:
            room = torch.empty(time_mix_workspace(table.chunks.shape[0], g), dtype=torch.uint8, device=out.device)
            ops.time_mix_chunks(proj, g, mix, cache.state, b.state_slots, b.cu_q, b.seq_lens, w.norm, eps, out, table, room)

    def forward(self, w: TimeMixWeights, cache: TimeMixState, inp, y, b, plan, small=None) -> None:
        T, n = b.num_tokens, w.geo.heads * w.geo.vp
        out = self.out[:T * n].view(T, n)
        self.mix(w, cache, inp, out, b, plan)
        ops.gemm(out, w.wo, out=y, out_f32=True)


class ForgetMixWeights:
    __slots__ = ("geo", "spec", "wproj", "bias", "lower", "norm", "wo")


class ForgetMixPart(Part):
    """Forget mixing beside another mixer (``parallel.py``), which makes the joint projection."""

    @staticmethod
    def geometry(spec: ForgetMixSpec) -> RecurrentGeometry:
        return RecurrentGeometry(spec.heads, spec.dim, spec.vdim, silu=True, gated=False, form="forget")

    @staticmethod
    def state_floats(spec) -> int:
        return ForgetMixPart.geometry(spec).state_floats

    def make(self, spec: ForgetMixSpec) -> ForgetMixWeights:
        g, f32 = self.geometry(spec), torch.float32
        if g.kp > MAX_DIM:
            raise ValueError(f"the recurrent kernels take up to {MAX_DIM} key channels per head")
        w = ForgetMixWeights()
        w.spec, w.geo, w.wproj = spec, g, None
        w.bias, w.lower = (self.zeros(g.heads * g.kp, dtype=f32) for _ in range(2))
        w.norm, w.wo = self.zeros(g.heads * g.vp, dtype=f32), self.zeros(self.r.wp, g.heads * g.vp)
        self.layers.append(w)
        return w

    def new_cache(self, w: ForgetMixWeights) -> RecurrentState:
        return RecurrentState.zeros(w.geo, self.r.scratch_state_slot + 1, self.r.device)

    def allocate(self) -> None:
        r, n = self.r, max(w.geo.heads * w.geo.kp for w in self.layers)
        self.keys, self.out = self.zeros(r.rows * 2 * n), self.zeros(r.rows * n)
        self.o = self.zeros(r.rows * n, dtype=torch.float32)

    def load(self, w: ForgetMixWeights, get, p: str) -> None:
        g, (_, _, ov, _) = w.geo, w.geo.offsets
        load_heads(w.wproj[:ov], get(p + "q"), g.heads, g.dim, g.kp)
        load_heads(w.wproj[ov:], get(p + "v"), g.heads, g.vdim, g.vp)
        load_head_vector(w.bias, get(p + "f.b").float(), g.heads, g.dim, g.kp)
        load_head_vector(w.lower, get(p + "lower").float(), g.heads, g.dim, g.kp)
        load_head_vector(w.norm, get(p + "norm").float().repeat(g.heads), g.heads, g.vdim, g.vp)
        load_head_columns(w.wo, get(p + "o"), g.heads, g.vdim, g.vp)

    def load_small(self, w: ForgetMixWeights, get, p: str, dst: torch.Tensor) -> None:
        load_heads(dst, get(p + "f"), w.geo.heads, w.geo.dim, w.geo.kp)

    plan = RecurrentPart.plan

    def mix(self, w: ForgetMixWeights, state: RecurrentState, proj, z, y, b, plan) -> None:
        """``y [T, wp]`` from the projected queries and values ``proj`` and the forget gate's logits ``z``."""
        T, n = b.num_tokens, w.geo.heads * w.geo.vp
        out = self.out[:T * n].view(T, n)
        self.recur(w, state, proj, z, out, b, plan)
        ops.gemm(out, w.wo, out=y, out_f32=True)

    def recur(self, w: ForgetMixWeights, state: RecurrentState, proj, z, out, b, plan) -> None:
        T, g, eps = b.num_tokens, w.geo, self.r.cfg.norm_eps
        n = g.heads * g.kp
        mix = ForgetMix(z, w.bias, w.lower, self.keys[:T * 2 * n].view(T, 2 * n))
        n_seq, rows, table = plan if time_mix_chunked_supported(g) else (b.rows, T, None)
        single = b.rows if b.cu_q is None else b.n_single
        if single > 0:
            ops.time_mix_decode(proj, g, mix, state, b.state_slots, b.seq_lens, w.norm, eps, out, single)
        if n_seq > single:
            o = self.o[:T * n].view(T, n)
            ops.recurrent_scan(proj, None, g, None, None, None, 1.0, state, b.state_slots, b.cu_q, b.seq_lens, o, rows, n_seq, single, mix=mix)
            ops.gated_norm(o[single:rows], w.norm, None, g, eps, out[single:], True)
        if table is not None:
            room = torch.empty(time_mix_workspace(table.chunks.shape[0], g), dtype=torch.uint8, device=out.device)
            ops.time_mix_chunks(proj, g, mix, state, b.state_slots, b.cu_q, b.seq_lens, w.norm, eps, out, table, room)


class DeltaWeights:
    __slots__ = ("geo", "spec", "wproj", "conv", "rate", "dt_bias", "norm", "wo")


@dataclass
class DeltaState:
    state: RecurrentState
    history: torch.Tensor | None     # [slots, taps - 1, channels], the last projected rows of every sequence, latest first


class DeltaPart(Part):
    """Gated delta rule: joint projection (queries, keys, values, output gate, logits of decay and step size), one kernel for the
    convolutions and the heads' units, the recurrence, norm and gate, output projection."""

    fuses_tail = True

    @staticmethod
    def geometry(spec: DeltaRuleSpec) -> RecurrentGeometry:
        return RecurrentGeometry(spec.heads, spec.dim, spec.vdim, silu=False, gated=False, form="delta", groups=spec.kv_heads)

    @staticmethod
    def state_floats(spec) -> int:
        g = DeltaPart.geometry(spec)
        return g.state_floats + (spec.taps - 1) * g.channels

    @staticmethod
    def small_rows(spec) -> int:
        return 2 * spec.heads

    def make(self, spec: DeltaRuleSpec, tail: int = 0) -> DeltaWeights:
        g, f32 = self.geometry(spec), torch.float32
        if max(g.kp, g.vp) > MAX_DIM or spec.taps > MAX_TAPS:
            raise ValueError(f"the delta rule's kernels take up to {MAX_DIM} key channels and value channels per head, convolutions of {MAX_TAPS}")
        w = DeltaWeights()
        w.spec, w.geo = spec, g
        w.wproj, w.wo = self.zeros(g.proj + tail, self.r.wp), self.zeros(self.r.wp, g.heads * g.vp)
        w.conv, w.norm = self.zeros(spec.taps, g.channels, dtype=f32), self.zeros(g.heads * g.vp, dtype=f32)
        w.rate, w.dt_bias = (self.zeros(g.heads, dtype=f32) for _ in range(2))
        self.layers.append(w)
        return w

    def new_cache(self, w: DeltaWeights) -> DeltaState:
        slots = self.r.scratch_state_slot + 1
        history = self.zeros(slots, w.spec.taps - 1, w.geo.channels) if w.spec.taps > 1 else None
        return DeltaState(RecurrentState.zeros(w.geo, slots, self.r.device), history)

    def allocate(self) -> None:
        r, f32, geos = self.r, torch.float32, {w.geo for w in self.layers}
        self.proj, self.rows = self.zeros(r.rows * max(g.proj for g in geos)), self.zeros(r.rows * max(g.channels for g in geos))
        self.units = self.zeros(r.rows * max(2 * g.key_heads for g in geos), dtype=f32)
        self.steps = self.zeros(r.rows * max(2 * g.heads for g in geos), dtype=f32)
        most = r.rows * max(g.heads * g.vp for g in geos)
        self.out, self.o = self.zeros(most), self.zeros(most, dtype=f32)

    def load(self, w: DeltaWeights, get, p: str) -> None:
        g = w.geo
        H, G, (_, ok, ov, og) = g.heads, g.key_heads, g.offsets
        for name, lo, hi, heads, dim, padded in (("q", 0, ok, G, g.dim, g.kp), ("k", ok, ov, G, g.dim, g.kp), ("v", ov, og, H, g.vdim, g.vp)):
            load_heads(w.wproj[lo:hi], get(p + name), heads, dim, padded)
            conv = get(f"{p}{name}.conv").float().T
            for t in range(w.spec.taps):
                load_head_vector(w.conv[t, lo:hi], conv[t].contiguous(), heads, dim, padded)
        load_heads(w.wproj[og:g.proj], get(p + "g"), H, g.vdim, g.vp)
        load_head_columns(w.wo, get(p + "o"), H, g.vdim, g.vp)
        load_head_vector(w.norm, get(p + "norm").float().repeat(H), H, g.vdim, g.vp)
        w.rate.copy_(get(p + "A_log").float().exp())
        w.dt_bias.copy_(get(p + "dt_bias").float())

    def load_small(self, w: DeltaWeights, get, p: str, dst: torch.Tensor) -> None:
        H, d = w.geo.heads, self.r.cfg.hidden_size
        dst[:H, :d].copy_(get(p + "b"))
        dst[H:2 * H, :d].copy_(get(p + "a"))

    plan = RecurrentPart.plan

    def _projected(self, w: DeltaWeights, T: int) -> torch.Tensor:
        return self.proj[:T * w.geo.proj].view(T, w.geo.proj)

    def project(self, w: DeltaWeights, inp, tail) -> None:
        ops.gemm(inp, w.wproj, out=self._projected(w, inp.shape[0]), tail=tail)

    def prepare(self, w: DeltaWeights, cache: DeltaState, small, b) -> tuple[torch.Tensor, DeltaRule]:
        """What the recurrence reads, after ``project``."""
        T, g = b.num_tokens, w.geo
        rows = self.rows[:T * g.channels].view(T, g.channels)
        rule = DeltaRule(self.units[:T * 2 * g.key_heads].view(T, -1), self.steps[:T * 2 * g.heads].view(T, -1))
        ops.delta_rows(self._projected(w, T), small, g, w.conv, cache.history, b.cu_q, b.positions, b.state_slots, w.rate, w.dt_bias, rows, rule)
        return rows, rule

    def recur(self, w: DeltaWeights, cache: DeltaState, rows, rule: DeltaRule, o, b, plan) -> None:
        T, g = b.num_tokens, w.geo
        n_seq, ends, table = plan if delta_chunked_supported(g) else (b.rows, T, None)
        args = (rows, None, g, None, None, None, 1.0, cache.state, b.state_slots)
        if b.n_single > 0:
            ops.recurrent_scan(*args, None, b.seq_lens, o, b.n_single, b.n_single, mix=rule)
        if n_seq > b.n_single:
            ops.recurrent_scan(*args, b.cu_q, b.seq_lens, o, ends, n_seq, b.n_single, mix=rule)
        if table is not None:
            room = torch.empty(delta_workspace(table.chunks.shape[0], g), dtype=torch.uint8, device=o.device)
            ops.delta_chunks(rows, g, rule, cache.state, b.state_slots, b.cu_q, b.seq_lens, o, table, room)

    def forward(self, w: DeltaWeights, cache: DeltaState, inp, y, b, plan, small=None) -> None:
        T, g = b.num_tokens, w.geo
        n = g.heads * g.vp
        o, out = self.o[:T * n].view(T, n), self.out[:T * n].view(T, n)
        rows, rule = self.prepare(w, cache, small, b)
        self.recur(w, cache, rows, rule, o, b, plan)
        ops.gated_norm(o, w.norm, self._projected(w, T)[:, g.offsets[3]:], g, self.r.cfg.norm_eps, out, True, silu=True)
        ops.gemm(out, w.wo, out=y, out_f32=True)

"""Grouped attention over cached keys and values (``ops/grouped.py``) as a part of a layer stack: one joint projection, one kernel for
the convolutions, norms, rotation and the cache append, attention with its head gate, the output projection. Sequences with one
new token take the decode kernel, portions the flash kernel, in one batch."""

from __future__ import annotations

import torch

from ... import ops
from ...models.stack import GroupedAttentionSpec
from ...ops.grouped import KV_BLOCK, MAX_HEAD, MAX_QK_CHANNELS, GroupedCache, GroupedGeometry
from .base import Part, load_head_columns, up


def grouped_geometry(m: GroupedAttentionSpec) -> GroupedGeometry:
    f = m.form
    return GroupedGeometry(m.heads, m.kv_heads, m.dim, m.vdim, m.taps, f.conv, f.norm, m.rot.dims, m.rot.interleaved,
                           m.size if f.span == "window" else 0, m.size if f.span == "chunk" else 0, f.temperature)


class GroupedWeights:
    __slots__ = ("geo", "spec", "wproj", "bproj", "wo", "conv", "q_norm", "k_norm", "temp", "table", "shared_projection")


class GroupedPart(Part):
    fuses_tail = True

    def __init__(self, runner):
        super().__init__(runner)
        self.tables: dict = {}

    @staticmethod
    def cache_row_elements(spec) -> int:
        g = grouped_geometry(spec)
        return 2 * g.kv_heads * g.dp

    @staticmethod
    def state_floats(spec) -> int:
        return grouped_geometry(spec).history

    @staticmethod
    def small_rows(spec) -> int:
        return spec.heads if spec.form.gate else 0

    def make(self, spec: GroupedAttentionSpec, tail: int = 0, output: bool = True, projection: bool = True) -> GroupedWeights:
        """``output``, ``projection``: with an output projection, a joint projection of its own (whoever else has it sets ``wproj`` and
        ``bproj`` and gives ``attend`` the projected rows)."""
        g, r, f32 = grouped_geometry(spec), self.r, torch.float32
        if g.dp > MAX_HEAD or g.v_col > MAX_QK_CHANNELS:
            raise ValueError(f"the attention kernels take heads of up to {MAX_HEAD} channels, queries and keys of {MAX_QK_CHANNELS} in all")
        w = GroupedWeights()
        w.spec, w.geo, w.shared_projection = spec, g, not projection
        w.wproj = self.zeros(g.proj + tail, r.wp) if projection else None
        w.bproj = self.zeros(g.proj + tail) if projection and spec.form.bias else None
        w.temp = self.zeros(g.heads, dtype=f32) if g.temperature else None
        w.wo = self.zeros(r.wp, g.heads * g.dp) if output else None
        w.conv = self.zeros(g.taps, g.channels, dtype=f32) if g.conv else None
        w.q_norm, w.k_norm = (self.zeros(n * g.dim, dtype=f32) if g.norm == "projection" else None for n in (g.heads, g.kv_heads))
        if spec.rot not in self.tables:
            self.tables[spec.rot] = ops.frequency_table(r.max_model_len, spec.rot.frequencies(), spec.rot.amplitude, r.device)
        w.table = self.tables[spec.rot]
        self.layers.append(w)
        return w

    def new_cache(self, w: GroupedWeights) -> GroupedCache:
        r, g = self.r, w.geo
        keys, values = (self.zeros(r.num_kv_blocks, g.kv_heads, KV_BLOCK, g.dp) for _ in range(2))
        return GroupedCache(keys, values, self.zeros(r.scratch_state_slot + 1, g.taps - 1, g.channels) if g.taps > 1 else None)

    def allocate(self) -> None:
        r, geos = self.r, {w.geo for w in self.layers}
        self.proj = self.zeros(r.rows * max([w.geo.proj for w in self.layers if not w.shared_projection], default=0))
        self.q = self.zeros(r.rows * max(g.heads * g.dp for g in geos))
        self.out = self.zeros(r.rows * max([w.geo.heads * w.geo.dp for w in self.layers if w.wo is not None], default=0))
        self.splits = {b: {g: ops.decode_num_splits(b, g.kv_heads, min(r.max_model_len, g.reach or r.max_model_len), head_dim=g.dp) if b <= 64 else 1
                           for g in geos} for b in sorted({*r.graph_batch_sizes, *range(1, min(r.max_batch, 64) + 1)})}
        need = max(ops.kv_workspace(g, b, n) for b, by in self.splits.items() for g, n in by.items())
        self.workspace = self.zeros(need, dtype=torch.float32) if r.bf16 else None

    def load(self, w: GroupedWeights, get, p: str) -> None:
        g, m, d = w.geo, w.spec, self.r.cfg.hidden_size
        for name, col, n in zip("qkv", (0, g.k_col, g.v_col), m.rows):
            w.wproj[col:col + n, :d].copy_(get(p + name))
            if w.bproj is not None:
                w.bproj[col:col + n].copy_(get(f"{p}{name}.b"))
            if g.conv:
                w.conv[:, col:col + n].copy_(get(f"{p}{name}.conv").float().T)
        if g.temperature:
            w.temp.copy_(get(p + "temp").float())
        if g.norm == "projection":
            w.q_norm.copy_(get(p + "q.norm").float())
            w.k_norm.copy_(get(p + "k.norm").float())
        if w.wo is not None:
            self.load_output(w, get, p, w.wo)

    def load_output(self, w: GroupedWeights, get, p: str, dst: torch.Tensor) -> None:
        load_head_columns(dst, get(p + "o"), w.geo.heads, w.geo.vdim, w.geo.dp)

    def load_small(self, w: GroupedWeights, get, p: str, dst: torch.Tensor) -> None:
        if w.spec.form.gate:
            dst[:w.geo.heads, :self.r.cfg.hidden_size].copy_(get(p + "g"))

    def plan(self, b):
        return self.splits.get(b.rows if b.cu_q is None else b.n_single, {})

    def _projected(self, w: GroupedWeights, T: int) -> torch.Tensor:
        return self.proj[:T * w.geo.proj].view(T, w.geo.proj)

    def project(self, w: GroupedWeights, inp, tail) -> None:
        ops.gemm(inp, w.wproj, bias=w.bproj, out=self._projected(w, inp.shape[0]), tail=tail)

    def attend(self, w: GroupedWeights, cache: GroupedCache, out, b, splits, small, factor: float = 1.0, proj=None) -> None:
        """Heads' outputs (gated, times ``factor``) into ``out [T, H * dp]``, after ``project`` (or from the rows ``proj``)."""
        T, g = b.num_tokens, w.geo
        q = self.q[:T * g.heads * g.dp].view(T, g.heads * g.dp)
        ops.grouped_append(self._projected(w, T) if proj is None else proj, g, conv=w.conv, cache=cache, cu_q=b.cu_q, positions=b.positions, state_slots=b.state_slots, slots=b.slots,
                           q_norm=w.q_norm, k_norm=w.k_norm, eps=self.r.cfg.norm_eps, table=w.table, q=q, q_factor=w.temp)
        ops.grouped_attention(q, g, cache, b.block_tables, b.cu_q, b.seq_lens, out, scale=w.spec.scale, rows=T, max_q=b.max_new, n_single=b.n_single,
                              gate=small if w.spec.form.gate else None, gate_scale=factor, workspace=self.workspace, splits=splits.get(g, 1))

    def forward(self, w: GroupedWeights, cache: GroupedCache, inp, y, b, plan, small=None) -> None:
        T, n = b.num_tokens, w.geo.heads * w.geo.dp
        out = self.out[:T * n].view(T, n)
        self.attend(w, cache, out, b, plan, small)
        ops.gemm(out, w.wo, out=y, out_f32=True)

"""Attention whose values are its keys (``ops/keyvalue.py``) as a part of a layer stack: one joint projection with biases
(queries, keys, output gate), one kernel for the query temperature and the cache append, attention with sink and gate, the
output projection. Sequences with one new token take the decode kernel, longer portions the flash kernel, in one batch."""

from __future__ import annotations

import torch

from ... import ops
from ...models.stack import KeyValueAttentionSpec
from ...ops.keyvalue import KV_BLOCK, KeyValueGeometry
from .base import Part, load_head_columns, load_head_vector, load_heads

MAX_HEAD = 512


def keyvalue_geometry(m: KeyValueAttentionSpec) -> KeyValueGeometry:
    return KeyValueGeometry(m.heads, m.kv_heads, m.dim)


class KeyValueWeights:
    __slots__ = ("geo", "spec", "wproj", "bproj", "wo", "bo", "sink")


class KeyValuePart(Part):
    fuses_tail = True

    @staticmethod
    def cache_row_elements(spec) -> int:
        g = keyvalue_geometry(spec)
        return g.kv_heads * g.dp

    def make(self, spec: KeyValueAttentionSpec, tail: int = 0) -> KeyValueWeights:
        g = keyvalue_geometry(spec)
        if g.dp > MAX_HEAD:
            raise ValueError(f"the attention kernels take heads of up to {MAX_HEAD} channels")
        w = KeyValueWeights()
        w.spec, w.geo = spec, g
        w.wproj, w.bproj = self.zeros(g.proj + tail, self.r.wp), self.zeros(g.proj + tail)
        w.wo, w.bo = self.zeros(self.r.wp, g.heads * g.dp), self.zeros(self.r.wp)
        w.sink = self.zeros(g.heads, dtype=torch.float32)
        self.layers.append(w)
        return w

    def new_cache(self, w):
        return self.zeros(self.r.num_kv_blocks, w.geo.kv_heads, KV_BLOCK, w.geo.dp)

    def allocate(self) -> None:
        r = self.r
        self.proj = self.zeros(r.rows * max(w.geo.proj for w in self.layers))
        self.out = self.zeros(r.rows * max(w.geo.heads * w.geo.dp for w in self.layers))
        self.splits = {b: {w.geo: ops.decode_num_splits(b, w.geo.kv_heads, r.max_model_len, head_dim=w.geo.dp) if b <= 64 else 1 for w in self.layers}
                       for b in sorted({*r.graph_batch_sizes, *range(1, min(r.max_batch, 64) + 1)})}
        need = max(ops.kv_workspace(g, b, n) for b, by in self.splits.items() for g, n in by.items())
        self.workspace = self.zeros(need, dtype=torch.float32) if r.bf16 else None

    def load(self, w: KeyValueWeights, get, p: str) -> None:
        g = w.geo
        H, G, D, d = g.heads, g.kv_heads, g.dim, g.dp
        load_heads(w.wproj[:g.k_col], get(p + "q"), H, D, d)
        load_heads(w.wproj[g.k_col:g.gate_col], get(p + "k"), G, D, d)
        load_heads(w.wproj[g.gate_col:g.proj], get(p + "g"), H, D, d)
        load_head_vector(w.bproj[:g.k_col], get(p + "q.b"), H, D, d)
        load_head_vector(w.bproj[g.k_col:g.gate_col], get(p + "k.b"), G, D, d)
        load_head_columns(w.wo, get(p + "o"), H, D, d)
        w.bo[:self.r.cfg.hidden_size].copy_(get(p + "o.b"))
        w.sink.copy_(get(p + "sink").float())

    def plan(self, b):
        single = b.rows if b.cu_q is None else b.n_single
        return self.splits.get(single, {})

    def _projected(self, w: KeyValueWeights, T: int) -> torch.Tensor:
        return self.proj[:T * w.geo.proj].view(T, w.geo.proj)

    def project(self, w: KeyValueWeights, inp, tail) -> None:
        ops.gemm(inp, w.wproj, bias=w.bproj, out=self._projected(w, inp.shape[0]), tail=tail)

    def forward(self, w: KeyValueWeights, cache, inp, y, b, splits, small=None) -> None:
        T, g, m = b.num_tokens, w.geo, w.spec
        proj = self._projected(w, T)
        out = self.out[:T * g.heads * g.dp].view(T, g.heads * g.dp)
        ops.kv_append(proj, g, b.positions, b.slots, m.q_temp.coef, m.q_temp.every, cache)
        ops.kv_attention(proj, g, cache, b.block_tables, b.cu_q, b.seq_lens, w.sink, out, scale=m.scale, rows=T, max_q=b.max_new,
                         n_single=b.n_single, workspace=self.workspace, splits=splits.get(g, 1))
        ops.gemm(out, w.wo, bias=w.bo, out=y, out_f32=True)

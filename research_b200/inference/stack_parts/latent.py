"""Latent attention (``ops/latent.py``) as a part of a layer stack.

One joint down projection (query latent, kv latent, rotated key part, gate logits), one fused norm / rotation / cache-append
kernel, the query up projection, attention, the output projection. Attention has two forms: on the cached latents themselves
for decoded tokens and portions of at most ``SHORT_PORTION`` tokens, on multiplied-out keys and values for longer portions.
Both kinds run in one packed batch.
"""

from __future__ import annotations

import torch

from ... import ops
from ...models.stack import LatentAttentionSpec
from ...ops.latent import LatentGeometry
from .base import Part

MAX_LATENT, MAX_CACHE_ROW = 1024, 1088
SHORT_PORTION = 16           # new tokens of a sequence up to which attention runs on the cached latents


def latent_geometry(m: LatentAttentionSpec) -> LatentGeometry:
    return LatentGeometry(m.heads, m.dim, m.rot_dim, m.rot.dims // 2, m.vdim, m.kv_rank, m.q_rank)


class LatentWeights:
    __slots__ = ("geo", "spec", "table", "wproj", "q_norm", "kv_norm", "wuq", "wuk", "wuv", "wo", "sink")


class GeometryBuffers:
    """Activations whose padding depends on a layer's geometry; layers of equal geometry share them."""

    def __init__(self, geo: LatentGeometry, rows: int, short_rows: int, dtype: torch.dtype, device: torch.device):
        H = geo.heads

        def zeros(*shape, dt=dtype):
            return torch.zeros(*shape, dtype=dt, device=device)

        self.cq = zeros(rows, geo.qp)
        self.gate = zeros(rows, H, dt=torch.float32)
        self.qn = zeros(H, short_rows, geo.dp)
        self.qa = zeros(H, short_rows, geo.cw)
        self.ol = zeros(H, short_rows, geo.rw)
        self.q = zeros(rows, H * (geo.dp + geo.rp))
        self.attn = zeros(rows, H * geo.vp)
        self.proj = zeros(rows, geo.proj, dt=torch.float32)


class LatentPart(Part):
    def __init__(self, runner):
        super().__init__(runner)
        self.tables: dict = {}

    @staticmethod
    def cache_row_elements(spec) -> int:
        return latent_geometry(spec).cw

    def make(self, spec: LatentAttentionSpec, tail: int = 0) -> LatentWeights:
        r, f32 = self.r, torch.float32
        g = latent_geometry(spec)
        if g.rw > MAX_LATENT or g.cw > MAX_CACHE_ROW:
            raise ValueError(f"the latent attention kernels take up to {MAX_LATENT} latent channels and cache rows of {MAX_CACHE_ROW}")
        w = LatentWeights()
        w.spec, w.geo = spec, g
        if spec.rot not in self.tables:
            self.tables[spec.rot] = ops.rope_table(r.max_model_len, spec.rot.dims, spec.rot.base, device=r.device, exact=True)
        w.table = self.tables[spec.rot]
        w.wproj = self.zeros(g.proj, r.wp)
        w.q_norm, w.kv_norm, w.sink = self.zeros(g.q_rank, dtype=f32), self.zeros(g.kv_rank, dtype=f32), self.zeros(g.heads, dtype=f32)
        w.wuq = self.zeros(g.heads * (g.dp + g.rp), g.qp)
        w.wuk = self.zeros(g.heads * g.dp, g.rw)
        w.wuv = self.zeros(g.heads * g.vp, g.rw)
        w.wo = self.zeros(r.wp, g.heads * g.vp)
        self.layers.append(w)
        return w

    def new_cache(self, w):
        return self.zeros(self.r.num_kv_blocks, ops.latent.LATENT_BLOCK, w.geo.cw)

    def allocate(self) -> None:
        r = self.r
        # multiplied-out keys and values need bf16 tensor-core tiles of a size the kernel has; otherwise (and in exact
        # mode) every token attends on the cached latents
        self.expand = (r.bf16 or not r.on_gpu) and all(ops.flash_latent_supported(w.geo) for w in self.layers)
        self.short_rows = min(r.rows, r.max_batch * SHORT_PORTION) if self.expand else r.rows
        self.bufs: dict[LatentGeometry, GeometryBuffers] = {}
        for w in self.layers:
            if w.geo not in self.bufs:
                self.bufs[w.geo] = GeometryBuffers(w.geo, r.rows, self.short_rows, r.dtype, r.device)
        self.workspace = ops.latent_workspace(list(self.bufs), r.device) if r.bf16 else None
        self.kinds = sorted({(w.geo, w.spec.window) for w in self.layers}, key=repr)    # layers that share an attention plan
        self.decode_plans = {k: torch.zeros(ops.latent_units(r.max_batch, k[0].heads, 1) + 1, dtype=torch.int32, device=r.device) for k in self.kinds}

    def load(self, w: LatentWeights, get, p: str) -> None:
        g, d = w.geo, self.r.cfg.hidden_size
        H, r0 = g.heads, g.q_rank
        r1 = r0 + g.kv_rank + g.rot_dim
        w.wproj[:r0, :d].copy_(get(p + "dq"))
        w.wproj[r0:r1, :d].copy_(get(p + "dkv"))
        w.wproj[r1:r1 + H, :d].copy_(get(p + "g"))
        w.q_norm.copy_(get(p + "dq.norm").float())
        w.kv_norm.copy_(get(p + "dkv.norm").float())
        w.sink.copy_(get(p + "sink").float())
        uq = get(p + "uq").view(H, g.dim + g.rot_dim, g.q_rank)
        wuq = w.wuq.view(H, g.dp + g.rp, g.qp)
        wuq[:, :g.dim, :g.q_rank].copy_(uq[:, :g.dim])
        wuq[:, g.dp:g.dp + g.rot_dim, :g.q_rank].copy_(uq[:, g.dim:])
        w.wuk.view(H, g.dp, g.rw)[:, :g.dim, :g.kv_rank].copy_(get(p + "uk").view(H, g.dim, g.kv_rank))
        w.wuv.view(H, g.vp, g.rw)[:, :g.vdim, :g.kv_rank].copy_(get(p + "uv").view(H, g.vdim, g.kv_rank))
        w.wo.view(-1, H, g.vp)[:d, :, :g.vdim].copy_(get(p + "o").view(d, H, g.vdim))

    # ------------------------------------------------------------------ one step
    def plan(self, b):
        """(rows on the cached latents, attention over them, attention over the rest)"""
        if b.cu_q is None:
            return b.num_tokens, self._short_attention(b.num_tokens, 1, None, b.seq_lens, b.block_tables, self.decode_plans), None
        lens = [b.host_cu_q[i + 1] - b.host_cu_q[i] for i in range(b.rows)]
        n_seq = b.rows                                      # sequences attending on the cached latents: a prefix of the batch
        if self.expand:
            n_seq = next((i for i, n in enumerate(lens) if n > SHORT_PORTION), b.rows)
            while b.host_cu_q[n_seq] > self.short_rows:     # (score() and other batches that are not ordered by length)
                n_seq -= 1
        n_short = b.host_cu_q[n_seq]
        short = None
        if n_short > 0:
            short = self._short_attention(n_short, max(lens[:n_seq], default=1), b.cu_q[:n_seq + 1], b.seq_lens[:n_seq], b.block_tables[:n_seq])
        return n_short, short, self._long_attention(b, n_seq, n_short) if n_seq < b.rows else None

    def forward(self, w: LatentWeights, cache, inp, y, b, plan, small=None) -> None:
        n_short, short_attn, long_attn = plan
        T, g, f = b.num_tokens, w.geo, self.bufs[w.geo]
        ops.gemm(inp, w.wproj, out=f.proj[:T], out_f32=True)
        ops.latent_append(f.proj[:T], g, w.q_norm, w.kv_norm, self.r.cfg.norm_eps, b.positions, b.slots, w.table, cache, f.cq, f.gate)
        q = ops.gemm(f.cq[:T], w.wuq, out=f.q[:T])
        ops.latent_query(q, g, b.positions, w.table, n_short, f.qn, f.qa)
        if n_short > 0:
            ops.head_gemm_absorb(f.qn, w.wuk, f.qa, n_short)
            short_attn(w, cache, f)
            ops.head_gemm_expand(f.ol, w.wuv, f.attn, n_short)
        if n_short < T:
            long_attn(w, cache, f)
        ops.gemm(f.attn[:T], w.wo, out=y, out_f32=True)

    def _short_attention(self, rows: int, max_q: int, cu_q, seq_lens, block_tables, plans: dict | None = None):
        """Attention on the cached latents for the first ``rows`` rows of the batch."""
        bf16 = self.r.bf16
        if bf16:
            n = seq_lens.shape[0]
            if plans is None:
                plans = {k: torch.empty(ops.latent_units(n, k[0].heads, max_q) + 1, dtype=torch.int32, device=self.r.device) for k in self.kinds}
            for (geo, window), plan in plans.items():
                ops.latent_plan(cu_q, seq_lens, geo, max_q, window, plan)

        def attend(w, cache, f):
            m = w.spec
            ops.latent_attention(f.qa, cache, w.geo, block_tables, cu_q, seq_lens, w.sink, f.gate, f.ol, scale=m.scale, window=m.window,
                                 rows=rows, max_q=max_q, plan=plans[(w.geo, m.window)] if bf16 else None, workspace=self.workspace)

        return attend

    def _long_attention(self, b, first: int, n_short: int):
        """Plan of the expanded form for the sequences ``first..``: per window, which cached rows they can see."""
        n_seq, dev, dt = b.rows - first, self.r.device, self.r.dtype
        plans: dict[int, tuple] = {}
        for win in {w.spec.window for w in self.layers}:
            lo, cu, most = [], [0], 0
            for i in range(first, b.rows):
                L, q = b.host_seq_lens[i], b.host_cu_q[i + 1] - b.host_cu_q[i]
                lo.append(max(0, L - q - win + 1))
                cu.append(cu[-1] + L - lo[-1])
                most = max(most, q)
            meta = torch.tensor(lo + cu, dtype=torch.int32).to(dev)
            plans[win] = (meta[:n_seq], meta[n_seq:], cu[-1], most)
        cu_q = b.cu_q[first:]

        def attend(w, cache, f):
            g, m = w.geo, w.spec
            k_lo, cu_k, n, max_q = plans[m.window]
            lat = torch.empty(n, g.rw, dtype=dt, device=dev)
            rot = torch.empty(n, g.rp, dtype=dt, device=dev)
            ops.latent_gather(cache, g, b.block_tables, first, cu_k, k_lo, n, lat, rot)
            k, v = ops.gemm(lat, w.wuk), ops.gemm(lat, w.wuv)
            ops.flash_latent_prefill(f.q, k, rot, v, g, cu_q, cu_k, w.sink, f.gate, f.attn, scale=m.scale, window=m.window,
                                     max_q=max_q, rows=b.num_tokens)

        return attend

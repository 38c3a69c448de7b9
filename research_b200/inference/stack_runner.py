"""Kernel-backed execution of layer-stack models (``LayerStackConfig``) over the engine's paged cache.

Step buffers, graph capture, packed batches and sampling come from ``RunnerBase``; this file has the weights, the cache
tensors and the layer sequence. The residual stream is fp32 with a copy in the activation type for the projections; a
sublayer reads the stream itself and its output is layer-normalised on the way back (the layer scale is folded into that
norm's weight and bias in fp32).

Per layer on the GPU: one joint down projection (query latent, kv latent, rotated key part, gate logits), one fused
norm / rotation / cache-append kernel, the query up projection, attention, the output projection, norm + residual, and
the feed-forward as gate|up with the clamped unit in the GEMM epilogue, down projection, norm + residual. Attention has
two forms (``ops/latent.py``): on the cached latents themselves for decoded tokens and portions of at most
``SHORT_PORTION`` tokens, on multiplied-out keys and values for longer portions. Both kinds run in one packed batch.

``dtype`` bf16 serves; fp32 runs the same sequence with every product in 32-bit.
"""

from __future__ import annotations

from collections.abc import Mapping

import torch

from .. import ops
from ..models.stack import ClampedGluSpec, LatentAttentionSpec, LayerStackConfig
from ..ops.latent import LatentGeometry, live_tables
from .model_runner import BLOCK, PackedBatch, RunnerBase

MAX_LATENT, MAX_CACHE_ROW = 1024, 1088
SHORT_PORTION = 16           # new tokens of a sequence up to which attention runs on the cached latents


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


def latent_geometry(m: LatentAttentionSpec) -> LatentGeometry:
    return LatentGeometry(m.heads, m.dim, m.rot_dim, m.rot.dims // 2, m.vdim, m.kv_rank, m.q_rank)


class StackLayer:
    """Padded device weights of one layer."""

    __slots__ = ("geo", "spec", "table", "wproj", "q_norm", "kv_norm", "wuq", "wuk", "wuv", "wo", "sink", "norm1", "norm2", "glu",
                 "wgu", "wd", "ffp", "cache")


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


class StackRunner(RunnerBase):
    supports_f32 = True
    joint_steps = True
    short_first = True

    def __init__(self, cfg: LayerStackConfig, weights: Mapping[str, torch.Tensor], *, device: torch.device, num_kv_blocks: int,
                 max_batch: int, max_model_len: int, max_prefill_tokens: int, use_cuda_graphs: bool = True,
                 graph_batch_sizes: tuple[int, ...] = (), tp=None, ep=None, dtype: torch.dtype = torch.bfloat16):
        if tp is not None or ep is not None:
            raise ValueError("layer-stack models run on one GPU per engine (no tensor or expert parallelism)")
        for x in cfg.layers:
            g = latent_geometry(x.mixer)
            if g.rw > MAX_LATENT or g.cw > MAX_CACHE_ROW:
                raise ValueError(f"the latent attention kernels take up to {MAX_LATENT} latent channels and cache rows of {MAX_CACHE_ROW}")
        self.tp = self.ep = None
        self.tp_size, self.tp_rank = 1, 0
        self._init_geometry(cfg, device=device, num_kv_blocks=num_kv_blocks, max_batch=max_batch, max_model_len=max_model_len,
                            max_prefill_tokens=max_prefill_tokens, use_cuda_graphs=use_cuda_graphs,
                            graph_batch_sizes=graph_batch_sizes, dtype=dtype)
        self.bf16 = self.on_gpu and dtype == torch.bfloat16
        d = cfg.hidden_size
        self.wp = _up(d, 8)
        self.vp = _up(cfg.vocab_size, 8)
        self.rows = max(max_prefill_tokens, max_batch)
        self.glu_bn = 256                               # tile width of the fused gate|up launch
        # multiplied-out keys and values need bf16 tensor-core tiles of a size the kernel has; otherwise (and in exact
        # mode) every token attends on the cached latents
        self.expand = (self.bf16 or not self.on_gpu) and all(ops.flash_latent_supported(latent_geometry(x.mixer)) for x in cfg.layers)
        self.short_rows = min(self.rows, max_batch * SHORT_PORTION) if self.expand else self.rows
        self._alloc_weights()
        self.load_weights(weights)
        self._init_step_buffers(self.vp)
        self._alloc_activations()

    @staticmethod
    def cache_bytes_per_block(cfg: LayerStackConfig, tp_size: int, dtype: torch.dtype) -> int:
        return sum(latent_geometry(x.mixer).cw for x in cfg.layers) * BLOCK * (4 if dtype == torch.float32 else 2)

    # ------------------------------------------------------------------ memory
    def _alloc_weights(self) -> None:
        cfg, dev, dt = self.cfg, self.device, self.dtype

        def zeros(*shape, dtype=dt):
            return torch.zeros(*shape, dtype=dtype, device=dev)

        f32 = torch.float32
        d = cfg.hidden_size
        self.embed = zeros(cfg.vocab_size, self.wp)
        self.head = zeros(self.vp, self.wp)
        self.final_norm = (zeros(d, dtype=f32), zeros(d, dtype=f32))
        tables: dict = {}
        self.layers: list[StackLayer] = []
        for spec in cfg.layers:
            m, g = spec.mixer, latent_geometry(spec.mixer)
            lw = StackLayer()
            lw.spec, lw.geo = spec, g
            if m.rot not in tables:
                tables[m.rot] = ops.rope_table(self.max_model_len, m.rot.dims, m.rot.base, device=dev, exact=True)
            lw.table = tables[m.rot]
            lw.wproj = zeros(g.proj, self.wp)
            lw.q_norm, lw.kv_norm, lw.sink = zeros(g.q_rank, dtype=f32), zeros(g.kv_rank, dtype=f32), zeros(g.heads, dtype=f32)
            lw.wuq = zeros(g.heads * (g.dp + g.rp), g.qp)
            lw.wuk = zeros(g.heads * g.dp, g.rw)
            lw.wuv = zeros(g.heads * g.vp, g.rw)
            lw.wo = zeros(self.wp, g.heads * g.vp)
            lw.norm1 = (zeros(d, dtype=f32), zeros(d, dtype=f32))
            lw.glu: ClampedGluSpec | None = spec.mlp
            lw.wgu = lw.wd = lw.norm2 = None
            lw.ffp = 0
            if spec.mlp is not None:
                lw.ffp = _up(spec.mlp.ff, self.glu_bn // 2 if self.bf16 else 8)
                lw.wgu, lw.wd = zeros(2 * lw.ffp, self.wp), zeros(self.wp, lw.ffp)
                lw.norm2 = (zeros(d, dtype=f32), zeros(d, dtype=f32))
            lw.cache = zeros(self.num_kv_blocks, BLOCK, g.cw)
            self.layers.append(lw)

    def _alloc_activations(self) -> None:
        dev, dt, n = self.device, self.dtype, self.rows
        d = self.cfg.hidden_size
        self.x = torch.zeros(n, d, dtype=torch.float32, device=dev)
        self.xb = torch.zeros(n, self.wp, dtype=dt, device=dev)
        self.y = torch.zeros(n, self.wp, dtype=torch.float32, device=dev)
        self.hl = torch.zeros(self.max_batch, self.wp, dtype=dt, device=dev)
        ffp = max([lw.ffp for lw in self.layers] + [8])
        self._gu = None if self.bf16 else torch.zeros(n * 2 * ffp, dtype=dt, device=dev)
        self._act = torch.zeros(n * ffp, dtype=dt, device=dev)
        self.bufs: dict[LatentGeometry, GeometryBuffers] = {}
        for lw in self.layers:
            if lw.geo not in self.bufs:
                self.bufs[lw.geo] = GeometryBuffers(lw.geo, n, self.short_rows, dt, dev)
        self.attn_ws = ops.latent_workspace(list(self.bufs), dev) if self.bf16 else None
        self.kinds = sorted({(lw.geo, lw.spec.mixer.window) for lw in self.layers}, key=repr)    # layers that share an attention plan
        self.decode_plans = {k: torch.zeros(ops.latent_units(self.max_batch, k[0].heads, 1) + 1, dtype=torch.int32, device=dev) for k in self.kinds}

    # ------------------------------------------------------------------ weights
    def load_weights(self, weights: Mapping[str, torch.Tensor]) -> None:
        """Copy checkpoint tensors into the padded buffers, in place (captured graphs stay valid)."""
        cfg, dev = self.cfg, self.device
        d = cfg.hidden_size

        def get(name: str) -> torch.Tensor:
            return weights[name].to(device=dev)

        def f32(name: str) -> torch.Tensor:
            return get(name).float()

        def norm_into(dst, name: str, scale: torch.Tensor | None) -> None:
            w, b = f32(name), f32(name + ".b")
            dst[0].copy_(w if scale is None else w * scale)
            dst[1].copy_(b if scale is None else b * scale)

        self.embed[:, :d].copy_(get("embed"))
        self.head[:cfg.vocab_size, :d].copy_(get("head"))
        norm_into(self.final_norm, "final.norm", None)
        for i, lw in enumerate(self.layers):
            p, g = f"l{i}.", lw.geo
            m = p + "mix."
            H, r0 = g.heads, g.q_rank
            r1 = r0 + g.kv_rank + g.rot_dim
            lw.wproj[:r0, :d].copy_(get(m + "dq"))
            lw.wproj[r0:r1, :d].copy_(get(m + "dkv"))
            lw.wproj[r1:r1 + H, :d].copy_(get(m + "g"))
            lw.q_norm.copy_(f32(m + "dq.norm"))
            lw.kv_norm.copy_(f32(m + "dkv.norm"))
            lw.sink.copy_(f32(m + "sink"))
            uq = get(m + "uq").view(H, g.dim + g.rot_dim, g.q_rank)
            wuq = lw.wuq.view(H, g.dp + g.rp, g.qp)
            wuq[:, :g.dim, :g.q_rank].copy_(uq[:, :g.dim])
            wuq[:, g.dp:g.dp + g.rot_dim, :g.q_rank].copy_(uq[:, g.dim:])
            lw.wuk.view(H, g.dp, g.rw)[:, :g.dim, :g.kv_rank].copy_(get(m + "uk").view(H, g.dim, g.kv_rank))
            lw.wuv.view(H, g.vp, g.rw)[:, :g.vdim, :g.kv_rank].copy_(get(m + "uv").view(H, g.vdim, g.kv_rank))
            lw.wo.view(self.wp, H, g.vp)[:d, :, :g.vdim].copy_(get(m + "o").view(d, H, g.vdim))
            norm_into(lw.norm1, p + "norm1", f32(p + "ls1"))
            if lw.glu is not None:
                gate, up = get(p + "mlp.gate"), get(p + "mlp.up")
                ff = lw.glu.ff
                if self.bf16:        # interleaved blocks for the fused epilogue; padding rows give 0
                    pad = torch.zeros(2, lw.ffp, self.wp, dtype=self.dtype, device=dev)
                    pad[0, :ff, :d], pad[1, :ff, :d] = gate, up
                    lw.wgu.copy_(ops.interleave_gate_up(pad[0], pad[1], self.glu_bn))
                else:
                    lw.wgu[:ff, :d].copy_(gate)
                    lw.wgu[lw.ffp:lw.ffp + ff, :d].copy_(up)
                lw.wd[:d, :ff].copy_(get(p + "mlp.down"))
                norm_into(lw.norm2, p + "norm2", f32(p + "ls2"))

    # ------------------------------------------------------------------ layers
    def _layers(self, T: int, tokens, positions, slots, n_short: int, short_attn, long_attn=None) -> None:
        """All layers over the first ``T`` rows. ``short_attn(lw, bufs)`` fills ``bufs.ol`` for the first ``n_short`` rows,
        ``long_attn(lw, bufs)`` the remaining rows of ``bufs.attn``."""
        eps = self.cfg.norm_eps
        x, xb, y = self.x[:T], self.xb[:T], self.y[:T]
        ops.embed_residual(tokens, self.embed, x, xb)
        for lw in self.layers:
            g, b = lw.geo, self.bufs[lw.geo]
            ops.gemm(xb, lw.wproj, out=b.proj[:T], out_f32=True)
            ops.latent_append(b.proj[:T], g, lw.q_norm, lw.kv_norm, eps, positions, slots, lw.table, lw.cache, b.cq, b.gate)
            q = ops.gemm(b.cq[:T], lw.wuq, out=b.q[:T])
            ops.latent_query(q, g, positions, lw.table, n_short, b.qn, b.qa)
            if n_short > 0:
                ops.head_gemm_absorb(b.qn, lw.wuk, b.qa, n_short)
                short_attn(lw, b)
                ops.head_gemm_expand(b.ol, lw.wuv, b.attn, n_short)
            if n_short < T:
                long_attn(lw, b)
            ops.gemm(b.attn[:T], lw.wo, out=y, out_f32=True)
            ops.layernorm_residual(y, lw.norm1[0], lw.norm1[1], eps, x, xb)
            if lw.glu is not None:
                act = self._act[:T * lw.ffp].view(T, lw.ffp)
                if self.bf16:
                    ops.gemm(xb, lw.wgu, out=act, bn=self.glu_bn, swiglu=True, glu_limit=lw.glu.limit)
                else:
                    gu = ops.gemm(xb, lw.wgu, out=self._gu[:T * 2 * lw.ffp].view(T, 2 * lw.ffp))
                    ops.clamped_glu(gu, lw.glu.limit, out=act)
                ops.gemm(act, lw.wd, out=y, out_f32=True)
                ops.layernorm_residual(y, lw.norm2[0], lw.norm2[1], eps, x, xb)

    def _head(self, h: torch.Tensor, logits: torch.Tensor) -> torch.Tensor:
        """``logits`` (rows padded to ``vp`` columns) of the final-normed rows ``h``, soft-capped."""
        cap = self.cfg.logit_softcap
        if self.bf16 and cap > 0:
            ops.gemm(h, self.head, out=logits, out_f32=True, softcap=cap)
        else:
            ops.gemm(h, self.head, out=logits, out_f32=True)
            if cap > 0:
                ops.softcap(logits, cap)
        return logits[:, :self.cfg.vocab_size]

    def _short_attention(self, rows: int, max_q: int, cu_q, seq_lens, block_tables, plans: dict | None = None):
        """Attention on the cached latents for the first ``rows`` rows of the batch."""
        if self.bf16:
            n = seq_lens.shape[0]
            if plans is None:
                plans = {k: torch.empty(ops.latent_units(n, k[0].heads, max_q) + 1, dtype=torch.int32, device=self.device) for k in self.kinds}
            for (geo, window), plan in plans.items():
                ops.latent_plan(cu_q, seq_lens, geo, max_q, window, plan)

        def attend(lw, b):
            m = lw.spec.mixer
            ops.latent_attention(b.qa, lw.cache, lw.geo, block_tables, cu_q, seq_lens, lw.sink, b.gate, b.ol, scale=m.scale, window=m.window,
                                 rows=rows, max_q=max_q, plan=plans[(lw.geo, m.window)] if self.bf16 else None, workspace=self.attn_ws)

        return attend

    # ------------------------------------------------------------------ decode
    def _decode_body(self, bk: int) -> None:
        self._layers(bk, self.d_tokens[:bk], self.d_pos[:bk], self.d_slots[:bk], bk,
                     self._short_attention(bk, 1, None, self.d_lens[:bk], self.bt_dev[:bk], self.decode_plans))
        ops.layernorm_rows(self.x[:bk], self.final_norm[0], self.final_norm[1], self.cfg.norm_eps, self.hl)
        logits = self._head(self.hl[:bk], self.logits_padded[:bk])
        self._sample(logits, self.d_temps[:bk], self.d_seeds[:bk], bk)

    def capture_graphs(self) -> None:
        super().capture_graphs()
        self._graph_tables = live_tables()        # tile tables whose addresses the graphs hold

    # ------------------------------------------------------------------ packed batches
    def _packed_forward(self, b: PackedBatch) -> torch.Tensor:
        T = b.num_tokens
        assert T <= self.rows, f"packed batch of {T} tokens, buffers hold {self.rows}"
        lens = [b.host_cu_q[i + 1] - b.host_cu_q[i] for i in range(b.rows)]
        n_seq = b.rows                                      # sequences attending on the cached latents: a prefix of the batch
        if self.expand:
            n_seq = next((i for i, n in enumerate(lens) if n > SHORT_PORTION), b.rows)
            while b.host_cu_q[n_seq] > self.short_rows:     # (score() and other batches that are not ordered by length)
                n_seq -= 1
        n_short = b.host_cu_q[n_seq]
        max_q = max(lens[:n_seq], default=1)
        short_attn = None
        if n_short > 0:
            short_attn = self._short_attention(n_short, max_q, b.cu_q[:n_seq + 1], b.seq_lens[:n_seq], b.block_tables[:n_seq])
        self._layers(T, b.tokens[:T], b.positions[:T], b.slots[:T], n_short, short_attn,
                     self._long_attention(b, n_seq, n_short) if n_seq < b.rows else None)
        return self.x[:T]

    def _long_attention(self, b: PackedBatch, first: int, n_short: int):
        """Plan of the expanded form for the sequences ``first..``: per window, which cached rows they can see."""
        n_seq = b.rows - first
        plans: dict[int, tuple] = {}
        for w in {lw.spec.mixer.window for lw in self.layers}:
            lo, cu, most = [], [0], 0
            for i in range(first, b.rows):
                L, q = b.host_seq_lens[i], b.host_cu_q[i + 1] - b.host_cu_q[i]
                lo.append(max(0, L - q - w + 1))
                cu.append(cu[-1] + L - lo[-1])
                most = max(most, q)
            meta = torch.tensor(lo + cu, dtype=torch.int32).to(self.device)
            plans[w] = (meta[:n_seq], meta[n_seq:], cu[-1], most)
        cu_q = b.cu_q[first:]

        def long_attn(lw, buf):
            g, m = lw.geo, lw.spec.mixer
            k_lo, cu_k, n, max_q = plans[m.window]
            lat = torch.empty(n, g.rw, dtype=self.dtype, device=self.device)
            rot = torch.empty(n, g.rp, dtype=self.dtype, device=self.device)
            ops.latent_gather(lw.cache, g, b.block_tables, first, cu_k, k_lo, n, lat, rot)
            k, v = ops.gemm(lat, lw.wuk), ops.gemm(lat, lw.wuv)
            ops.flash_latent_prefill(buf.q, k, rot, v, g, cu_q, cu_k, lw.sink, buf.gate, buf.attn, scale=m.scale, window=m.window,
                                     max_q=max_q, rows=b.num_tokens)

        return long_attn

    def _row_logits(self, x, rows) -> torch.Tensor:
        n = rows.numel()
        h = self.hl if n <= self.max_batch else torch.zeros(n, self.wp, dtype=self.dtype, device=self.device)
        ops.layernorm_rows(x, self.final_norm[0], self.final_norm[1], self.cfg.norm_eps, h, rows)
        return self._head(h[:n], torch.empty(n, self.vp, dtype=torch.float32, device=self.device))

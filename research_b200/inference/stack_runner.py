"""Kernel-backed execution of layer-stack models (``LayerStackConfig``) over the engine's paged cache and state slots.

Step buffers, graph capture, packed batches and sampling come from ``RunnerBase``, mixers and feed-forwards from
``stack_parts``; this file puts layers together. The residual stream is fp32; projections read activations in the serving
type. Three kinds of layer (``Design.block``):

* post_norm: a sublayer reads the stream itself (a copy in the activation type) and its output is layer-normalised on the way
  back; the layer scale is folded into that norm's weight and bias in fp32;
* parallel: mixer and feed-forward read one RMS norm of the stream; the residual add, the sum over a token's experts and
  the next layer's norm are one kernel. A per-layer token input (``TokenSideSpec``) enters between the add and that norm: two narrow
  products over the stream, and its own norm in the same kernel as the next layer's;
* sandwich: every sublayer reads a norm of the stream, and a norm of its output is added. The weighing of a sublayer's parts (experts, two
  mixers under norms of their own), the norm behind it, the residual add and the next sublayer's norm are one kernel.

Looped layers run several times with the same weights; every run has a cache or state of its own, and a pass starts with a
product that mixes the embedding output into the stream.

``dtype`` bf16 serves; fp32 runs the same sequence with every product in 32-bit.
"""

from __future__ import annotations

from collections.abc import Mapping
from dataclasses import dataclass
from typing import Any

import torch

from .. import ops
from ..models.stack import ExpertsSpec, LayerSpec, LayerStackConfig
from ..ops.latent import live_tables
from .model_runner import BLOCK, PackedBatch, RunnerBase
from .stack_parts import FEED_FORWARD_PARTS, MIXER_PARTS
from .stack_parts.base import Part, up


class StackLayer:
    """Weights of one layer: those of its mixer and feed-forward parts, the norms, the narrow fp32 projection."""

    __slots__ = ("spec", "mixer", "mix", "feed_forward", "ff", "norm1", "norm2", "wsmall", "wsmall_ff", "mix_small", "side", "norm1b", "norm2b")


@dataclass
class SideWeights:
    """Per-layer token input: the gate ``[sp, wp]``, the projection back ``[wp, sp]``, the norm's weight, the layer's columns of the side
    embedding."""

    gate: torch.Tensor
    proj: torch.Tensor
    norm: torch.Tensor
    col: int


@dataclass
class StackRun:
    """One execution of a layer in a step, with the cache or state that belongs to it."""

    layer: StackLayer
    cache: Any
    enters: bool


def _mixer_part(spec: LayerSpec):
    return MIXER_PARTS[type(spec.mixer)]


class StackRunner(RunnerBase):
    supports_f32 = True
    joint_steps = True
    short_first = True

    def __init__(self, cfg: LayerStackConfig, weights: Mapping[str, torch.Tensor], *, device: torch.device, num_kv_blocks: int,
                 max_batch: int, max_model_len: int, max_prefill_tokens: int, use_cuda_graphs: bool = True,
                 graph_batch_sizes: tuple[int, ...] = (), tp=None, ep=None, dtype: torch.dtype = torch.bfloat16):
        if tp is not None or ep is not None:
            raise ValueError("layer-stack models run on one GPU per engine (no tensor or expert parallelism)")
        self.tp = self.ep = None
        self.tp_size, self.tp_rank = 1, 0
        cfg = cfg.fitted(weights)
        self._init_geometry(cfg, device=device, num_kv_blocks=num_kv_blocks, max_batch=max_batch, max_model_len=max_model_len,
                            max_prefill_tokens=max_prefill_tokens, use_cuda_graphs=use_cuda_graphs,
                            graph_batch_sizes=graph_batch_sizes, dtype=dtype)
        self.bf16 = self.on_gpu and dtype == torch.bfloat16
        self.parallel, self.sandwich = cfg.design.block == "parallel", cfg.design.block == "sandwich"
        if not self.sandwich and any(isinstance(x.mlp, ExpertsSpec) and (x.mlp.identity or x.mlp.routing.shared_gate) for x in cfg.layers):
            raise ValueError("identity experts and gated shared experts belong to sandwich blocks")
        self.wp = up(cfg.hidden_size, 8)
        self.vp = up(cfg.vocab_size, 8)
        self.rows = max(max_prefill_tokens, max_batch)
        self.parts: dict[type, Part] = {}
        self._alloc_weights()
        self.load_weights(weights)
        self._init_step_buffers(self.vp)
        self._alloc_activations()

    @staticmethod
    def cache_bytes_per_block(cfg: LayerStackConfig, tp_size: int, dtype: torch.dtype) -> int:
        rows = sum(_mixer_part(cfg.layers[x.layer]).cache_row_elements(cfg.layers[x.layer].mixer) for x in cfg.runs)
        return rows * BLOCK * (4 if dtype == torch.float32 else 2)

    @staticmethod
    def state_bytes_per_slot(cfg: LayerStackConfig, dtype: torch.dtype) -> int:
        return 4 * sum(_mixer_part(cfg.layers[x.layer]).state_floats(cfg.layers[x.layer].mixer) for x in cfg.runs)

    # ------------------------------------------------------------------ memory
    def _part(self, cls: type) -> Part:
        if cls not in self.parts:
            self.parts[cls] = cls(self)
        return self.parts[cls]

    def _alloc_weights(self) -> None:
        cfg, dev, dt = self.cfg, self.device, self.dtype

        def zeros(*shape, dtype=dt):
            return torch.zeros(*shape, dtype=dtype, device=dev)

        def norm():
            vectors = [zeros(self.wp, dtype=torch.float32) for _ in range(2)]
            if not self.sandwich:
                return tuple(vectors)
            return ops.StreamNorm(*vectors, zeros(1, dtype=torch.float32)) if cfg.design.bounded_norms else ops.StreamNorm(vectors[0])

        # (a tied head reads the embedding table itself, whose rows are padded like the head's)
        self.embed = zeros(self.vp, self.wp)
        self.head = self.embed if cfg.design.tied else zeros(self.vp, self.wp)
        self.final_norm = norm()
        self.loop_in = zeros(self.wp, 2 * self.wp) if cfg.loop is not None else None
        self.side_dim = cfg.token_side.dim if cfg.token_side is not None else 0
        self.sp = up(self.side_dim, 8)
        self.side_embed = zeros(cfg.vocab_size, cfg.num_layers * self.side_dim) if self.side_dim else None
        self.layers: list[StackLayer] = []
        for spec in cfg.layers:
            lw = StackLayer()
            lw.spec = spec
            lw.mixer = self._part(_mixer_part(spec))
            lw.norm1, lw.norm2 = norm(), None
            lw.norm1b = lw.norm2b = norm() if self.sandwich else None
            lw.feed_forward = lw.ff = None
            lw.mix_small = up(lw.mixer.small_rows(spec.mixer), 8)
            ff_small = 0
            if spec.mlp is not None:
                lw.feed_forward = self._part(FEED_FORWARD_PARTS[type(spec.mlp)])
                lw.ff = lw.feed_forward.make(spec.mlp)
                lw.norm2 = None if self.parallel else norm()
                lw.norm2b = norm() if self.sandwich else None
                ff_small = up(lw.feed_forward.small_rows(spec.mlp), 8)
            # the mixer's gate logits and, where both read the same activations, the router
            n = lw.mix_small + (ff_small if self.parallel else 0)
            lw.mix = lw.mixer.make(spec.mixer, n)
            lw.wsmall = None if n == 0 else lw.mix.wproj[-n:] if lw.mixer.fuses_tail else zeros(n, self.wp)
            lw.wsmall_ff = None if ff_small == 0 else lw.wsmall[lw.mix_small:] if self.parallel else zeros(ff_small, self.wp)
            lw.side = SideWeights(zeros(self.sp, self.wp), zeros(self.wp, self.sp), zeros(self.wp, dtype=torch.float32),
                                  len(self.layers) * self.side_dim) if self.side_dim else None
            self.layers.append(lw)
        self.runs = [StackRun(self.layers[x.layer], self.layers[x.layer].mixer.new_cache(self.layers[x.layer].mix), x.enters) for x in cfg.runs]

    def _alloc_activations(self) -> None:
        dev, dt, n = self.device, self.dtype, self.rows
        self.x = torch.zeros(n, self.wp, dtype=torch.float32, device=dev)
        self.xb = torch.zeros(n, self.wp, dtype=dt, device=dev)          # what the sublayers read
        self.y = torch.zeros(n, self.wp, dtype=torch.float32, device=dev)
        self.y2 = torch.zeros(n, self.wp, dtype=torch.float32, device=dev)
        self.hl = torch.zeros(self.max_batch, self.wp, dtype=dt, device=dev)
        self.x_loop = torch.zeros(n, 2 * self.wp, dtype=dt, device=dev) if self.loop_in is not None else None     # stream | embedding output
        self.side_z = torch.zeros(n, self.sp, dtype=torch.float32, device=dev)
        self.side_a = torch.zeros(n, self.sp, dtype=dt, device=dev)
        most = max([w.shape[0] for lw in self.layers for w in (lw.wsmall, lw.wsmall_ff) if w is not None], default=0)
        self._small = torch.zeros(n * most, dtype=torch.float32, device=dev)
        for part in self.parts.values():
            part.allocate()

    # ------------------------------------------------------------------ weights
    def load_weights(self, weights: Mapping[str, torch.Tensor]) -> None:
        """Copy checkpoint tensors into the padded buffers, in place (captured graphs stay valid)."""
        cfg, dev = self.cfg, self.device
        d = cfg.hidden_size

        def get(name: str) -> torch.Tensor:
            return weights[name].to(device=dev)

        def f32(name: str) -> torch.Tensor:
            return get(name).float()

        def norm_into(dst, name: str, scale: torch.Tensor | None = None) -> None:
            if self.sandwich:
                dst.weight[:d].copy_(f32(name) + float(cfg.design.unit_norms))
                if dst.alpha is not None:
                    dst.bias[:d].copy_(f32(name + ".b"))
                    dst.alpha.copy_(f32(name + ".alpha").reshape(1))
                return
            if self.parallel:          # RMS norm
                dst[0][:d].copy_(f32(name) + float(cfg.design.unit_norms))
                return
            w, b = f32(name), f32(name + ".b")
            dst[0][:d].copy_(w if scale is None else w * scale)
            dst[1][:d].copy_(b if scale is None else b * scale)

        self.embed[:cfg.vocab_size, :d].copy_(get("embed"))
        if not cfg.design.tied:
            self.head[:cfg.vocab_size, :d].copy_(get("head"))
        if self.loop_in is not None:
            w = get("loop.in")
            self.loop_in[:d, :d].copy_(w[:, :d])
            self.loop_in[:d, self.wp:self.wp + d].copy_(w[:, d:])
        if self.side_embed is not None:
            self.side_embed.copy_(get("side.embed"))
        norm_into(self.final_norm, "final.norm")
        for i, lw in enumerate(self.layers):
            p = f"l{i}."
            lw.mixer.load(lw.mix, get, p + "mix.")
            scaled = not (self.parallel or self.sandwich)
            norm_into(lw.norm1, p + "norm1", f32(p + "ls1") if scaled else None)
            if self.sandwich:
                norm_into(lw.norm1b, p + "norm1b")
            if lw.mix_small:
                lw.mixer.load_small(lw.mix, get, p + "mix.", lw.wsmall[:lw.mix_small])
            if lw.ff is not None:
                lw.feed_forward.load(lw.ff, get, p + "mlp.")
                if lw.wsmall_ff is not None:
                    lw.feed_forward.load_small(lw.ff, get, p + "mlp.", lw.wsmall_ff)
                if not self.parallel:
                    norm_into(lw.norm2, p + "norm2", f32(p + "ls2") if scaled else None)
                if self.sandwich:
                    norm_into(lw.norm2b, p + "norm2b")
            if lw.side is not None:
                lw.side.gate[:self.side_dim, :d].copy_(get(p + "side.gate"))
                lw.side.proj[:d, :self.side_dim].copy_(get(p + "side.proj"))
                lw.side.norm[:d].copy_(f32(p + "side.norm"))

    # ------------------------------------------------------------------ layers
    def _small_rows(self, inp: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """The narrow projections of ``inp``, fp32."""
        return ops.gemm(inp, w, out=self._small_buffer(inp.shape[0], w), out_f32=True)

    def _small_buffer(self, T: int, w: torch.Tensor) -> torch.Tensor:
        return self._small[:T * w.shape[0]].view(T, w.shape[0])

    def _project(self, lw: StackLayer, inp: torch.Tensor) -> torch.Tensor | None:
        """The mixer's projections; returns the narrow fp32 one."""
        if lw.wsmall is None or lw.mixer.fuses_tail:
            small = self._small_buffer(inp.shape[0], lw.wsmall) if lw.wsmall is not None else None
            lw.mixer.project(lw.mix, inp, small)
            return small
        lw.mixer.project(lw.mix, inp, None)
        return self._small_rows(inp, lw.wsmall)

    def _layers(self, b: PackedBatch) -> None:
        """All layer runs over the batch's rows; leaves the residual stream in ``self.x``."""
        plans = {part: part.planned(b) for part in self.parts.values()}
        if self.parallel:
            self._parallel_layers(b, plans)
        elif self.sandwich:
            self._sandwich_layers(b, plans)
        else:
            self._post_norm_layers(b, plans)

    def _enter_pass(self, T: int) -> None:
        """``x = W [x; embedding output]``: a pass of the loop begins (the stream's copy is in ``x_loop`` already)."""
        ops.gemm(self.x_loop[:T], self.loop_in, out=self.x[:T], out_f32=True)

    def _embed(self, b: PackedBatch, first_copy: torch.Tensor | None) -> None:
        """Embedding output into the stream, its second half of ``x_loop`` and, if given, another copy."""
        x0 = self.x_loop[:, self.wp:] if self.x_loop is not None else None
        ops.stream_embed(b.tokens[:b.num_tokens], self.embed[:self.cfg.vocab_size], self.cfg.hidden_size, self.x, x0, first_copy)

    def _parallel_layers(self, b: PackedBatch, plans: dict) -> None:
        T, d, eps, m = b.num_tokens, self.cfg.hidden_size, self.cfg.norm_eps, self.cfg.residual_mult
        x, h, y = self.x[:T], self.xb[:T], self.y[:T]
        xl = self.x_loop[:T, :self.wp] if self.x_loop is not None else None
        self._embed(b, xl)
        add: dict = {}                                 # what the layer before leaves for the stream
        for run in self.runs:
            lw = run.layer
            if run.enters:
                if add:
                    ops.stream_norm(x, d, **add, mult=m, eps=eps, copy=xl)
                    add = {}
                self._enter_pass(T)
            ops.stream_norm(x, d, **add, mult=m, weight=lw.norm1[0], eps=eps, h=h)
            small = self._project(lw, h)
            lw.mixer.forward(lw.mix, run.cache, h, y, b, plans[lw.mixer], small)
            add = {"y1": y}
            if lw.ff is not None:
                add.update(lw.feed_forward.forward(lw.ff, h, self.y2[:T], small[:, lw.mix_small:] if small is not None else None))
            if lw.side is not None:
                ops.stream_norm(x, d, **add, mult=m, copy=h)
                self._token_side(lw.side, b, h, y)
                add = {"side": y, "side_weight": lw.side.norm}
        ops.stream_norm(x, d, **add, mult=m, eps=eps)

    def _sandwich_layers(self, b: PackedBatch, plans: dict) -> None:
        T, d, eps = b.num_tokens, self.cfg.hidden_size, self.cfg.norm_eps
        x, h, y = self.x[:T], self.xb[:T], self.y[:T]
        xl = self.x_loop[:T, :self.wp] if self.x_loop is not None else None
        self._embed(b, xl)
        add: dict = {}                                 # what the sublayer before leaves for the stream, and the norm behind it

        def left_by(parts: dict | None, norm) -> dict:
            parts = dict(parts) if parts else {"y1": y}
            return {"y": parts.pop("y1", None) if "y1" in parts else parts.pop("y2", None), "post": norm, **parts}

        for run in self.runs:
            lw = run.layer
            if run.enters:
                if add:
                    ops.stream_sandwich(x, d, **add, eps=eps, copy=xl)
                    add = {}
                self._enter_pass(T)
            ops.stream_sandwich(x, d, **add, pre=lw.norm1, eps=eps, h=h)
            small = self._project(lw, h)
            add = left_by(lw.mixer.forward(lw.mix, run.cache, h, y, b, plans[lw.mixer], small), lw.norm1b)
            if lw.ff is not None:
                ops.stream_sandwich(x, d, **add, pre=lw.norm2, eps=eps, h=h)
                small = self._small_rows(h, lw.wsmall_ff) if lw.wsmall_ff is not None else None
                add = left_by(lw.feed_forward.forward(lw.ff, h, y, small), lw.norm2b)
        ops.stream_sandwich(x, d, **add, eps=eps)

    def _token_side(self, w: SideWeights, b: PackedBatch, xb: torch.Tensor, y: torch.Tensor) -> None:
        """``y = W_proj (gelu_tanh(W_gate x) * e)`` with the layer's part ``e`` of the tokens' side embedding."""
        T = b.num_tokens
        z, a = self.side_z[:T], self.side_a[:T]
        ops.gemm(xb, w.gate, out=z, out_f32=True)
        ops.token_side(z, b.tokens[:T], self.side_embed, w.col, a, self.side_dim)
        ops.gemm(a, w.proj, out=y, out_f32=True)

    def _post_norm_layers(self, b: PackedBatch, plans: dict) -> None:
        T, d, eps = b.num_tokens, self.cfg.hidden_size, self.cfg.norm_eps
        x, xb, y = self.x[:T], self.xb[:T], self.y[:T]
        self._embed(b, xb)
        for run in self.runs:
            lw = run.layer
            if run.enters:
                ops.stream_norm(x, d, copy=self.x_loop[:T, :self.wp])
                self._enter_pass(T)
                ops.stream_norm(x, d, copy=xb)
            small = self._project(lw, xb)
            lw.mixer.forward(lw.mix, run.cache, xb, y, b, plans[lw.mixer], small)
            ops.layernorm_residual(y, lw.norm1[0], lw.norm1[1], eps, x, xb, d)
            if lw.ff is not None:
                small = self._small_rows(xb, lw.wsmall_ff) if lw.wsmall_ff is not None else None
                add = lw.feed_forward.forward(lw.ff, xb, y, small)
                if "experts" in add:
                    y.zero_()
                    ops.stream_norm(y, d, **add)
                ops.layernorm_residual(y, lw.norm2[0], lw.norm2[1], eps, x, xb, d)

    def _final_rows(self, x: torch.Tensor, out: torch.Tensor, rows: torch.Tensor | None = None) -> None:
        d, eps = self.cfg.hidden_size, self.cfg.norm_eps
        if self.sandwich:
            ops.stream_sandwich(x, d, pre=self.final_norm, eps=eps, h=out, rows=rows)
        elif self.parallel:
            ops.stream_norm(x, d, weight=self.final_norm[0], eps=eps, h=out, rows=rows)
        else:
            ops.layernorm_rows(x, self.final_norm[0], self.final_norm[1], eps, out, rows, d)

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

    # ------------------------------------------------------------------ decode
    def _decode_batch(self, bk: int) -> PackedBatch:
        return PackedBatch(rows=bk, num_tokens=bk, padded=bk, max_new=1, tokens=self.d_tokens[:bk], positions=self.d_pos[:bk], slots=self.d_slots[:bk],
                           cu_q=None, seq_lens=self.d_lens[:bk], block_tables=self.bt_dev[:bk], host_cu_q=[], host_seq_lens=[],
                           state_slots=self.d_state_slots[:bk], n_single=bk)

    def _decode_body(self, bk: int) -> None:
        self._layers(self._decode_batch(bk))
        self._final_rows(self.x[:bk], self.hl)
        logits = self._head(self.hl[:bk], self.logits_padded[:bk])
        self._sample(logits, self.d_temps[:bk], self.d_seeds[:bk], bk)

    def capture_graphs(self) -> None:
        super().capture_graphs()
        self._graph_tables = live_tables()        # tile tables whose addresses the graphs hold

    # ------------------------------------------------------------------ packed batches
    def _packed_forward(self, b: PackedBatch) -> torch.Tensor:
        T = b.num_tokens
        assert T <= self.rows, f"packed batch of {T} tokens, buffers hold {self.rows}"
        b.tokens, b.positions, b.slots = b.tokens[:T], b.positions[:T], b.slots[:T]
        self._layers(b)
        return self.x[:T]

    def _row_logits(self, x, rows) -> torch.Tensor:
        n = rows.numel()
        h = self.hl if n <= self.max_batch else torch.zeros(n, self.wp, dtype=self.dtype, device=self.device)
        self._final_rows(x, h, rows)
        return self._head(h[:n], torch.empty(n, self.vp, dtype=torch.float32, device=self.device))

"""Routed experts on one GPU (``csrc/moe_sm100.cu`` routing and row movement, grouped GEMMs) with a PyTorch twin.

A router's logits -> the ``top`` largest softmax or sigmoid scores, divided by their sum or not; rows are gathered expert by
expert (times their weight, when it belongs to the input), the gated unit runs as two grouped products (tile tables made on the
device, so the layer fits a CUDA graph) and the second one stores every result row at its ``(token, choice)`` place. The
weighted sum over the choices is left to whoever adds the result to the residual stream (``elementwise.stream_norm``).

Choices from ``experts`` on (``identity`` of them) are no experts: they get no rows, and the sum takes the layer's input with their
weight. A correction per choice may decide together with the score, without entering the weight.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle
from .elementwise import clamped_glu, clamped_glu_reference
from .gemm import EPI_STORE, RbGemmArgs, _lib as _gemm_lib, _lib_f32, interleave_gate_up

c_int, c_ll, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_void_p
MAX_EXPERTS, MAX_TOP = 256, 32


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


def _lib() -> ctypes.CDLL:
    lib = _native.load("rb_moe")
    if not getattr(lib, "_rb_experts_typed", False):
        lib.rb_experts_route.argtypes = [c_vp, c_ll, c_vp] + [c_int] * 6 + [c_vp] * 4
        lib.rb_experts_plan.argtypes = [c_vp, c_int, c_vp, c_int, c_int, c_vp, c_vp, c_int, c_int, c_vp, c_vp, c_int, c_vp, c_vp, c_vp]
        lib.rb_experts_gather.argtypes = [c_vp, c_ll, c_vp] + [c_int] * 5 + [c_vp] * 4 + [c_ll, c_int, c_vp, c_int, c_vp, c_vp]
        for f in ("rb_experts_route", "rb_experts_plan", "rb_experts_gather"):
            getattr(lib, f).restype = c_int
        lib._rb_experts_typed = True
    return lib


@dataclass(frozen=True)
class ExpertsGeometry:
    experts: int
    top: int
    ff: int
    width: int           # padded row width of the stream
    limit: float | None  # of the clamped unit; None: silu(gate) * up
    bn: int              # tile width of the grouped products (gate and up rows are interleaved in halves of it when it is fused)
    fused: bool          # the unit runs in the first product's epilogue
    scores: str = "softmax"
    normalize: bool = True
    scale_input: bool = False    # a choice's weight multiplies the expert's input, not its output
    identity: int = 0            # choices that hand the input on

    @property
    def choices(self) -> int:
        return self.experts + self.identity

    @property
    def ffp(self) -> int:
        return _up(self.ff, self.bn // 2 if self.fused else 8)

    @staticmethod
    def make(experts: int, top: int, ff: int, width: int, limit: float | None, dtype: torch.dtype, scores: str = "softmax", normalize: bool = True,
             scale_input: bool = False, identity: int = 0) -> "ExpertsGeometry":
        if experts + identity > MAX_EXPERTS or top > MAX_TOP:
            raise ValueError(f"the expert kernels take up to {MAX_EXPERTS} experts, {MAX_TOP} per token")
        return ExpertsGeometry(experts, top, ff, width, limit, 128 if dtype == torch.bfloat16 else 64, dtype == torch.bfloat16, scores, normalize,
                               scale_input, identity)


class ExpertsScratch:
    """Routing tables, gathered rows and tile tables for up to ``rows`` tokens; layers of equal geometry share one."""

    def __init__(self, geo: ExpertsGeometry, rows: int, dtype: torch.dtype, device: torch.device):
        def buf(*shape, dt=dtype):
            return torch.zeros(*shape, dtype=dt, device=device)

        i32, E, k, cap = torch.int32, geo.experts, geo.top, rows * geo.top
        self.cap = cap
        self.idx, self.w = buf(rows, k, dt=i32), buf(rows, k, dt=torch.float32)
        self.y = buf(cap, geo.width)
        if device.type != "cuda":
            return
        self.counts, self.cursor, self.offsets = buf(E, dt=i32), buf(2 * E, dt=i32), buf(E + 1, dt=i32)
        self.xp, self.act, self.ret = buf(cap, geo.width), buf(cap, geo.ffp), buf(cap, dt=torch.int64)
        self.gu = None if geo.fused else buf(cap, 2 * geo.ffp)
        self.max_tiles = (cap // 128 + min(E, cap) + 1) * max(-(-2 * geo.ffp // geo.bn), -(-geo.width // geo.bn))
        self.tiles_gu, self.tiles_dn, self.ntiles = buf(self.max_tiles, 4, dt=i32), buf(self.max_tiles, 4, dt=i32), buf(2, dt=i32)


def pack_experts(gates, ups, downs, geo: ExpertsGeometry, wgu: torch.Tensor, wd: torch.Tensor) -> None:
    """Copy one layer's expert matrices (iterables of ``[ff, d]``, ``[ff, d]``, ``[d, ff]``) into the stacked padded buffers
    ``wgu [E*2*ffp, width]``, ``wd [E*width, ffp]``."""
    ffp = geo.ffp
    gu3, wd3 = wgu.view(geo.experts, 2 * ffp, -1), wd.view(geo.experts, geo.width, ffp)
    for e, (g, u, dn) in enumerate(zip(gates, ups, downs)):
        pad = torch.zeros(2, ffp, geo.width, dtype=wgu.dtype, device=wgu.device)
        pad[0, :geo.ff, :g.shape[1]], pad[1, :geo.ff, :u.shape[1]] = g, u
        gu3[e].copy_(interleave_gate_up(pad[0], pad[1], geo.bn) if geo.fused else pad.view(2 * ffp, -1))
        wd3[e, :dn.shape[0], :geo.ff].copy_(dn)


def route_reference(logits: torch.Tensor, top: int, scores: str = "softmax", normalize: bool = True,
                    correction: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    s = logits.float().softmax(-1) if scores == "softmax" else torch.sigmoid(logits.float())
    idx = (s if correction is None else s + correction).topk(top, -1).indices
    w = s.gather(-1, idx)
    return idx.to(torch.int32), w / (w.sum(-1, keepdim=True) + 1e-20) if normalize else w


def _grouped(a, b, c, geo: ExpertsGeometry, sc: ExpertsScratch, group_n: int, K: int, tiles, count, unit: bool, row_dst) -> None:
    if not geo.fused:
        rc = _lib_f32().rb_gemm_f32_grouped(a.data_ptr(), b.data_ptr(), c.data_ptr(), K, a.stride(0), b.stride(0), c.stride(0), tiles.data_ptr(),
                                            count.data_ptr(), sc.max_tiles, group_n, row_dst.data_ptr() if row_dst is not None else None,
                                            stream_handle(a.device))
        check_rc(rc, "rb_gemm_f32_grouped")
        return
    args = RbGemmArgs()
    args.A[0], args.B[0], args.C = a.data_ptr(), b.data_ptr(), c.data_ptr()
    args.lda, args.ldb, args.ldc = a.stride(0), b.stride(0), c.stride(0)
    args.M, args.N, args.K = a.shape[0], b.shape[0], K
    args.a_parts = args.b_parts = 1
    args.bn, args.epi_mode = geo.bn, EPI_STORE
    args.rank, args.world = 0, 1
    args.status = status_tensor(a.device).data_ptr()
    args.tile_table, args.num_tiles_ptr = tiles.data_ptr(), count.data_ptr()
    args.group_n, args.max_tiles = group_n, sc.max_tiles
    if unit:
        args.swiglu, args.glu_kind, args.glu_limit = 1, int(geo.limit is not None), geo.limit or 0.0
    args.row_dst = row_dst.data_ptr() if row_dst is not None else None
    check_rc(_gemm_lib().rb_gemm_bf16_ex(ctypes.byref(args), stream_handle(a.device)), "rb_gemm_bf16_ex(experts)")


def experts_plan(logits, geo: ExpertsGeometry, sc: ExpertsScratch, correction=None) -> None:
    """Choices and weights of every token, the experts' row ranges and the tile tables of both products."""
    T, s, st = logits.shape[0], stream_handle(logits.device), ptr(status_tensor(logits.device))
    check_rc(_lib().rb_experts_route(ptr(logits), logits.stride(0), ptr(correction), T, geo.choices, geo.experts, geo.top, int(geo.scores == "sigmoid"), int(geo.normalize), ptr(sc.idx),
                                     ptr(sc.w), ptr(sc.counts), s), "rb_experts_route")
    check_rc(_lib().rb_experts_plan(ptr(sc.counts), geo.experts, ptr(sc.offsets), 2 * geo.ffp, geo.bn, ptr(sc.tiles_gu), ptr(sc.ntiles), geo.width,
                                    geo.bn, ptr(sc.tiles_dn), sc.ntiles.data_ptr() + 4, sc.max_tiles, ptr(sc.cursor), st, s), "rb_experts_plan")


def experts_gather(h, geo: ExpertsGeometry, sc: ExpertsScratch) -> None:
    es = h.element_size()
    check_rc(_lib().rb_experts_gather(ptr(h), h.stride(0) * es, ptr(sc.idx), h.shape[0], geo.top, geo.width * es, geo.experts, geo.choices, ptr(sc.cursor), ptr(sc.xp),
                                      ptr(sc.ret), ptr(sc.y), geo.width * es, sc.cap, ptr(sc.w) if geo.scale_input else None, int(es == 4),
                                       ptr(status_tensor(h.device)), stream_handle(h.device)),
             "rb_experts_gather")


def experts_up(geo: ExpertsGeometry, sc: ExpertsScratch, wgu, T: int) -> None:
    dst = sc.act if geo.fused else sc.gu
    _grouped(sc.xp, wgu, dst, geo, sc, 2 * geo.ffp, geo.width, sc.tiles_gu, sc.ntiles, geo.fused, None)
    if not geo.fused:
        clamped_glu(sc.gu[:T * geo.top], geo.limit, out=sc.act[:T * geo.top])


def experts_down(geo: ExpertsGeometry, sc: ExpertsScratch, wd) -> None:
    _grouped(sc.act, wd, sc.y, geo, sc, geo.width, geo.ffp, sc.tiles_dn, sc.ntiles[1:], False, sc.ret)


def experts_forward(h, logits, geo: ExpertsGeometry, sc: ExpertsScratch, wgu, wd, correction=None) -> tuple[torch.Tensor, torch.Tensor | None]:
    """Results ``[T * top, width]`` of every token's chosen experts and the weights ``[T, top]`` they are still to be multiplied by
    (None with ``scale_input``) for ``h [T, width]`` and the router's logits ``[T, >= choices]`` (fp32). ``correction [choices]``: see
    above. The choices are left in ``sc.idx``; rows of choices that are no experts hold nothing."""
    T, k = h.shape[0], geo.top
    assert T * k <= sc.cap and logits.dtype == torch.float32
    if h.is_cuda:
        experts_plan(logits, geo, sc, correction)
        experts_gather(h, geo, sc)
        experts_up(geo, sc, wgu, T)
        experts_down(geo, sc, wd)
        return sc.y[:T * k], None if geo.scale_input else sc.w[:T]
    idx, w = route_reference(logits[:, :geo.choices], k, geo.scores, geo.normalize, correction)
    sc.idx[:T], sc.w[:T] = idx, w
    y = sc.y[:T * k].view(T, k, geo.width)
    gu3, wd3 = wgu.view(geo.experts, 2 * geo.ffp, -1), wd.view(geo.experts, geo.width, geo.ffp)
    for e in range(geo.experts):
        tok, slot = (idx == e).nonzero(as_tuple=True)
        if tok.numel():
            x = h[tok].float() * w[tok, slot, None] if geo.scale_input else h[tok].float()
            y[tok, slot] = (clamped_glu_reference(x @ gu3[e].float().T, geo.limit) @ wd3[e].float().T).to(y.dtype)
    return sc.y[:T * k], None if geo.scale_input else sc.w[:T]

"""Attention whose values are its keys (one cached row per token and kv head), with grouped query heads, a query
temperature, a softmax sink and an element-wise output gate. Kernels: ``csrc/attn_sm100.cu`` (decode, exact mode, append),
``csrc/flash_sm100.cu`` (long portions); the CPU twins are here too.

Cache per layer: ``[num_blocks, G, 16, dp]``. The joint projection of a token is ``q [H, dp] | k [G, dp] | gate [H, dp]``.
"""

from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p
KV_BLOCK = 16
_DT = {torch.bfloat16: 0, torch.float32: 1}


@dataclass(frozen=True)
class KeyValueGeometry:
    heads: int
    kv_heads: int
    dim: int

    @property
    def dp(self) -> int:
        return -(-self.dim // 64) * 64

    @property
    def proj(self) -> int:
        return (2 * self.heads + self.kv_heads) * self.dp

    @property
    def k_col(self) -> int:
        return self.heads * self.dp

    @property
    def gate_col(self) -> int:
        return (self.heads + self.kv_heads) * self.dp

    @property
    def tensor_core(self) -> bool:       # head sizes the tensor-core kernels are built for
        return self.dp in (64, 128)


def _lib() -> ctypes.CDLL:
    lib = _native.load("rb_attn")
    if not getattr(lib, "_rb_kv_typed", False):
        lib.rb_kv_append.argtypes = [c_vp, c_ll, c_vp, c_vp, c_float, c_int, c_vp] + [c_int] * 6 + [c_vp, c_vp]
        gate = [c_vp, c_ll, c_vp, c_ll, c_float]
        lib.rb_kv_decode.argtypes = [c_vp, c_ll] + [c_vp] * 5 + gate + [c_vp, c_ll, c_vp] + [c_int] * 10 + [c_float, c_vp, c_vp]
        lib.rb_kv_simple.argtypes = [c_vp, c_ll] + [c_vp] * 6 + gate + [c_vp, c_ll] + [c_int] * 11 + [c_float, c_vp, c_vp]
        lib.rb_kv_gate.argtypes = [c_vp, c_vp, c_vp, c_vp, c_ll] + [c_int] * 5 + [c_vp]
        for f in ("rb_kv_append", "rb_kv_decode", "rb_kv_simple", "rb_kv_gate"):
            getattr(lib, f).restype = c_int
        lib._rb_kv_typed = True
    return lib


def kv_append(proj, geo: KeyValueGeometry, positions, slots, coef: float, every: int, cache) -> None:
    """Queries times ``1 + coef ln(floor((p + 1) / every) + 1)`` in place; keys -> the cache rows at ``slots`` (negative: skipped)."""
    T, H, G, D = proj.shape[0], geo.heads, geo.kv_heads, geo.dp
    if not proj.is_cuda:
        temp = 1 + coef * torch.log(torch.div(positions.long() + 1, every, rounding_mode="floor").float() + 1)
        proj[:, :H * D] = (proj[:, :H * D].float() * temp[:, None]).to(proj.dtype)
        ok = slots >= 0
        sl = slots[ok].long()
        cache[sl // KV_BLOCK, :, sl % KV_BLOCK] = proj[ok][:, geo.k_col:geo.gate_col].view(-1, G, D)
        return
    assert proj.stride(1) == 1 and cache.is_contiguous()
    rc = _lib().rb_kv_append(ptr(proj), proj.stride(0), ptr(positions), ptr(slots), coef, every, ptr(cache), cache.shape[0], H, G, D, T,
                             _DT[proj.dtype], ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_kv_append")


def kv_attention_reference(proj, geo: KeyValueGeometry, cache, block_tables, cu_q, seq_lens, sink, out, scale: float) -> None:
    H, G, D = geo.heads, geo.kv_heads, geo.dp
    for b in range(seq_lens.shape[0]):
        t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
        L = int(seq_lens[b])
        if L == 0 or t1 == t0:
            out[t0:t1] = 0
            continue
        key = torch.arange(L)
        kv = cache[block_tables[b, key // KV_BLOCK].long(), :, key % KV_BLOCK].float().repeat_interleave(H // G, 1)
        s = torch.einsum("thd,khd->htk", proj[t0:t1, :H * D].view(-1, H, D).float(), kv) * scale
        pos = torch.arange(L - (t1 - t0), L)
        s = s.masked_fill((key[None] > pos[:, None])[None], -math.inf)
        p = torch.cat([s, sink.view(H, 1, 1).expand(H, t1 - t0, 1)], -1).softmax(-1)[..., :-1]
        o = torch.einsum("htk,khd->thd", p, kv).reshape(t1 - t0, H * D)
        out[t0:t1] = (o * torch.sigmoid(proj[t0:t1, geo.gate_col:].float())).to(out.dtype)


def kv_attention(proj, geo: KeyValueGeometry, cache, block_tables, cu_q, seq_lens, sink, out, *, scale: float, rows: int, max_q: int,
                 n_single: int, workspace=None, splits: int = 1) -> None:
    """Causal attention of the packed new tokens in ``proj`` (after ``kv_append``) against the cached rows:
    ``out [T, H*dp] = sigmoid(gate) * softmax-with-sink(q k^T scale) k``.

    The first ``n_single`` sequences have one new token each and go to the decode kernel (``splits`` key ranges per
    sequence, ``workspace`` of ``kv_workspace`` floats); ``cu_q`` None: all of them."""
    if not proj.is_cuda:
        kv_attention_reference(proj[:rows], geo, cache, block_tables, cu_q, seq_lens, sink, out, scale)
        return
    H, G, D, B, dev = geo.heads, geo.kv_heads, geo.dp, seq_lens.shape[0], proj.device
    assert cache.is_contiguous() and block_tables.stride(1) == 1 and out.is_contiguous() and sink.dtype == torch.float32
    gate = (proj.data_ptr() + proj.element_size() * geo.gate_col, proj.stride(0), None, 0, 1.0)
    if proj.dtype == torch.float32 or not geo.tensor_core:
        rc = _lib().rb_kv_simple(ptr(proj), proj.stride(0), ptr(cache), None, ptr(block_tables), ptr(cu_q), ptr(seq_lens), ptr(sink), *gate, ptr(out),
                                 out.stride(0), H, G, D, block_tables.stride(0), cache.shape[0], B, rows, max_q, 0, 0, _DT[proj.dtype], scale,
                                 ptr(status_tensor(dev)), stream_handle(dev))
        check_rc(rc, "rb_kv_simple")
        return
    if cu_q is None:
        n_single = B
    if n_single > 0:
        rc = _lib().rb_kv_decode(ptr(proj), proj.stride(0), ptr(cache), None, ptr(block_tables), ptr(seq_lens), ptr(sink), *gate, ptr(out),
                                 out.stride(0), ptr(workspace), n_single, H, G, D, block_tables.stride(0), cache.shape[0], KV_BLOCK, splits, 0, 0, scale,
                                 ptr(status_tensor(dev)), stream_handle(dev))
        check_rc(rc, "rb_kv_decode", 2 if splits > 1 else 1)
    if n_single < B:
        from .flash import flash_paged_prefill

        lse = torch.empty(H, rows, dtype=torch.float32, device=dev)
        flash_paged_prefill(proj[:rows, :H * D].view(rows, H, D), cache, cache, block_tables[n_single:], cu_q[n_single:], seq_lens[n_single:], max_q,
                            scale, 0, out.view(-1, H, D)[:rows], lse)
        rc = _lib().rb_kv_gate(ptr(out), ptr(lse), ptr(sink), proj.data_ptr() + 2 * geo.gate_col, proj.stride(0), H, D, n_single, rows - n_single, rows,
                               stream_handle(dev))
        check_rc(rc, "rb_kv_gate")


def kv_workspace(geo: KeyValueGeometry, batch: int, splits: int) -> int:
    """Floats the split decode needs for its partial results."""
    return batch * geo.heads * splits * (geo.dp + 2)

"""Attention with grouped heads over cached keys and values: short convolutions on the projections, norms and rotation of queries
and keys, a factor per query head, a window or chunks, a gate per head. Kernels: ``csrc/attn_sm100.cu`` (append, decode, exact mode),
``csrc/flash_sm100.cu`` (portions); the CPU twins are here too.

The joint projection of a token is ``q [H, dim] | k [G, dim] | v [G, vdim]`` (each part padded to 8 columns); the append kernel
pads heads to ``dp`` channels on its way to the query buffer ``[T, H * dp]`` and to the caches ``[num_blocks, G, 16, dp]``.
"""

from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle
from .keyvalue import KV_BLOCK, _DT, _lib as _kv_lib

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p
MAX_HEAD = 512
MAX_QK_CHANNELS = 51200          # projected channels of queries and keys that one CTA keeps in shared memory
NORMS = {"": 0, "projection": 1, "head": 2}


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


@dataclass(frozen=True)
class GroupedGeometry:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int = 1                    # of the convolution; 1: a factor per channel
    conv: bool = False
    norm: str = ""                   # "projection" (before the rotation, with weights), "head" (after it), ""
    rot_dims: int = 0
    interleaved: bool = False
    window: int = 0                  # keys a query sees: the last so many (0: all)
    chunk: int = 0                   # or those of its own run of so many positions
    temperature: bool = False        # queries times a number of their head

    @property
    def dp(self) -> int:
        return _up(max(self.dim, self.vdim), 64)

    @property
    def k_col(self) -> int:
        return _up(self.heads * self.dim, 8)

    @property
    def v_col(self) -> int:
        return self.k_col + _up(self.kv_heads * self.dim, 8)

    @property
    def channels(self) -> int:       # projected channels, padding included
        return self.v_col + _up(self.kv_heads * self.vdim, 8)

    @property
    def proj(self) -> int:           # columns of the joint projection (the narrow fp32 one starts behind them)
        return _up(self.channels, 32)

    @property
    def history(self) -> int:        # channels of look-back a sequence keeps
        return (self.taps - 1) * self.channels

    @property
    def tensor_core(self) -> bool:   # head sizes the tensor-core kernels are built for
        return self.dp in (64, 128)

    @property
    def reach(self) -> int:          # most keys a query can see (0: no bound)
        return self.window or self.chunk


@dataclass
class GroupedCache:
    keys: torch.Tensor               # [num_blocks, G, 16, dp]
    values: torch.Tensor
    history: torch.Tensor | None     # [slots, taps - 1, channels], the last projected values of every sequence, latest first


class GroupedAppendArgs(ctypes.Structure):
    _fields_ = ([(n, c_vp) for n in ("proj", "conv", "hist", "cu_q", "positions", "state_slots", "slots", "q_norm", "k_norm", "q_factor", "table", "q",
                                     "keys", "values", "status")] + [("ld", c_ll)]
                + [(n, c_int) for n in ("k_col", "v_col", "channels", "taps", "B", "num_state_slots", "norm", "half", "interleaved", "max_pos",
                                        "num_blocks", "H", "G", "dim", "vdim", "DP", "T", "dtype")] + [("eps", c_float)])


def _lib() -> ctypes.CDLL:
    lib = _kv_lib()
    if not getattr(lib, "_rb_grouped_typed", False):
        lib.rb_grouped_append.argtypes, lib.rb_grouped_append.restype = [ctypes.POINTER(GroupedAppendArgs), c_vp], c_int
        lib._rb_grouped_typed = True
    return lib


def _flash_lib() -> ctypes.CDLL:
    lib = _native.load("rb_flash")
    if not getattr(lib, "_rb_grouped_typed", False):
        lib.rb_flash_fwd_ex.argtypes = ([c_vp] * 4 + [c_ll] + [c_vp] * 5 + [c_int] * 15 + [c_vp, c_ll, c_float, c_float, c_vp, c_vp])
        lib.rb_flash_fwd_ex.restype = c_int
        lib._rb_grouped_typed = True
    return lib


def first_key(geo: GroupedGeometry, position):
    """First key a query at ``position`` (int or tensor) sees."""
    if geo.window:
        first = position - geo.window + 1
        return first.clamp(min=0) if torch.is_tensor(first) else max(first, 0)
    return position - position % geo.chunk if geo.chunk else position * 0


def look_back(rows: torch.Tensor, depth: int, history, cu_q, positions, state_slots) -> torch.Tensor:
    """``[T, depth, C]``: the rows 1 .. depth places before every packed row, from the batch or the sequences' ``history [slots, depth,
    C]`` (latest first), zeros in front of a sequence. CPU twin of what the kernels do on the way."""
    T, C = rows.shape
    out = rows.new_zeros(T, depth, C)
    n_seq = T if cu_q is None else cu_q.numel() - 1
    for b in range(n_seq):
        t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
        if t1 == t0 or int(state_slots[b]) < 0:
            continue
        past = history[int(state_slots[b])].flip(0).clone()
        past[:max(depth - int(positions[t0]), 0)] = 0            # (another sequence's, before this one's first token)
        line = torch.cat([past, rows[t0:t1]])
        for d in range(1, depth + 1):
            out[t0:t1, d - 1] = line[depth - d:depth - d + t1 - t0]
    return out


def move_history(rows: torch.Tensor, history, cu_q, state_slots) -> None:
    """CPU twin: ``history`` of the batch's sequences after their new rows."""
    depth = history.shape[1]
    for b in range(rows.shape[0] if cu_q is None else cu_q.numel() - 1):
        t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
        slot = int(state_slots[b])
        if slot >= 0 and t1 > t0:
            history[slot] = torch.cat([history[slot].flip(0), rows[t0:t1]])[-depth:].flip(0)


def _rotate(x, cs, interleaved: bool):
    """``x [T, h, d]`` with the pairs of its first channels turned by ``cs [T, half, 2]``."""
    half = cs.shape[1]
    a, b = (slice(0, 2 * half, 2), slice(1, 2 * half, 2)) if interleaved else (slice(0, half), slice(half, 2 * half))
    c, s, out = cs[:, None, :, 0], cs[:, None, :, 1], x.clone()
    out[..., a], out[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
    return out


def _append_reference(proj, geo, conv, cache, cu_q, positions, state_slots, slots, q_norm, k_norm, eps, table, q, q_factor) -> None:
    T, H, G, D, E = proj.shape[0], geo.heads, geo.kv_heads, geo.dim, geo.vdim
    u = proj[:, :geo.channels].float()
    x = u * conv[geo.taps - 1] if geo.conv else u
    if geo.taps > 1:
        raw = proj[:, :geo.channels]
        back = look_back(raw, geo.taps - 1, cache.history, cu_q, positions, state_slots).float()
        x = x + sum(conv[geo.taps - 1 - d] * back[:, d - 1] for d in range(1, geo.taps))
        move_history(raw, cache.history, cu_q, state_slots)
    qk = []
    for x0, n, w in ((x[:, :H * D], H, q_norm), (x[:, geo.k_col:geo.k_col + G * D], G, k_norm)):
        if geo.norm == "projection":
            x0 = x0 * torch.rsqrt(x0.pow(2).mean(-1, keepdim=True) + eps) * w
        x0 = _rotate(x0.reshape(T, n, D), table[positions.long()], geo.interleaved)
        if geo.norm == "head":
            x0 = x0 * torch.rsqrt(x0.pow(2).mean(-1, keepdim=True) + eps)
        qk.append(x0)
    if q_factor is not None:
        qk[0] = qk[0] * q_factor[:, None]
    q3 = q[:T].view(T, H, geo.dp)
    q3.zero_()
    q3[..., :D] = qk[0].to(q.dtype)
    ok = slots >= 0
    sl = slots[ok].long()
    cache.keys[sl // KV_BLOCK, :, sl % KV_BLOCK, :D] = qk[1][ok].to(q.dtype)
    v = x[:, geo.v_col:geo.v_col + G * E].reshape(T, G, E)
    cache.values[sl // KV_BLOCK, :, sl % KV_BLOCK, :E] = v[ok].to(q.dtype)


def grouped_append(proj, geo: GroupedGeometry, *, conv, cache: GroupedCache, cu_q, positions, state_slots, slots, q_norm, k_norm, eps: float, table,
                   q, q_factor=None) -> None:
    """From the joint projection ``proj [T, >= channels]`` of the packed new tokens: convolved, normed and rotated queries into
    ``q [T, H * dp]``, keys and values into the cache rows ``slots`` (negative: skipped). ``conv [taps, channels]`` fp32, latest tap
    last; ``table [positions, rot_dims / 2, 2]``; ``state_slots [B]`` own the convolution's look back, which moves on; queries times
    ``q_factor [H]`` (fp32, or None)."""
    T = proj.shape[0]
    if not proj.is_cuda:
        _append_reference(proj, geo, conv, cache, cu_q, positions, state_slots, slots, q_norm, k_norm, eps, table, q, q_factor)
        return
    assert proj.stride(1) == 1 and q.is_contiguous() and cache.keys.is_contiguous() and cache.values.is_contiguous() and table.is_contiguous()
    a = GroupedAppendArgs()
    assert (conv is not None) == geo.conv and (geo.conv or geo.taps == 1)
    for name, t in (("proj", proj), ("conv", conv), ("hist", cache.history), ("cu_q", cu_q), ("positions", positions), ("state_slots", state_slots),
                    ("slots", slots), ("q_norm", q_norm), ("k_norm", k_norm), ("q_factor", q_factor), ("table", table), ("q", q), ("keys", cache.keys),
                    ("values", cache.values), ("status", status_tensor(proj.device))):
        setattr(a, name, t.data_ptr() if t is not None else None)
    a.ld, a.k_col, a.v_col, a.channels, a.taps = proj.stride(0), geo.k_col, geo.v_col, geo.channels, geo.taps
    a.B, a.num_state_slots = (T if cu_q is None else cu_q.numel() - 1), (cache.history.shape[0] if cache.history is not None else 0)
    a.norm, a.half, a.interleaved, a.max_pos = NORMS[geo.norm], geo.rot_dims // 2, int(geo.interleaved), table.shape[0]
    a.num_blocks, a.H, a.G, a.dim, a.vdim, a.DP = cache.keys.shape[0], geo.heads, geo.kv_heads, geo.dim, geo.vdim, geo.dp
    a.T, a.dtype, a.eps = T, _DT[proj.dtype], eps
    check_rc(_lib().rb_grouped_append(ctypes.byref(a), stream_handle(proj.device)), "rb_grouped_append", 2 if cu_q is not None and geo.taps > 1 else 1)


def _attention_reference(q, geo, cache, block_tables, cu_q, seq_lens, gate, gate_scale, out, scale) -> None:
    H, G, D = geo.heads, geo.kv_heads, geo.dp
    for b in range(seq_lens.shape[0]):
        t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
        L = int(seq_lens[b])
        if L == 0 or t1 == t0:
            out[t0:t1] = 0
            continue
        key = torch.arange(L)
        k, v = (c[block_tables[b, key // KV_BLOCK].long(), :, key % KV_BLOCK].float().repeat_interleave(H // G, 1) for c in (cache.keys, cache.values))
        s = torch.einsum("thd,khd->htk", q[t0:t1].view(-1, H, D).float(), k) * scale
        pos = torch.arange(L - (t1 - t0), L)
        s = s.masked_fill((key[None] > pos[:, None]) | (key[None] < first_key(geo, pos)[:, None]), -math.inf)
        o = torch.einsum("htk,khd->thd", s.softmax(-1), v) * gate_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[t0:t1, :H].float())[..., None]
        out[t0:t1] = o.reshape(t1 - t0, H * D).to(out.dtype)


def grouped_attention(q, geo: GroupedGeometry, cache: GroupedCache, block_tables, cu_q, seq_lens, out, *, scale: float, rows: int, max_q: int,
                      n_single: int, gate=None, gate_scale: float = 1.0, workspace=None, splits: int = 1) -> None:
    """Attention of the packed new tokens ``q [rows, H * dp]`` (after ``grouped_append``) over the cached keys they see, into
    ``out [rows, H * dp]`` (any row stride), times ``gate_scale`` and, with ``gate [rows, >= H]`` (fp32), its sigmoid per head.

    The first ``n_single`` sequences have one new token each and go to the decode kernel (``splits`` key ranges per sequence,
    ``workspace`` of ``kv_workspace`` floats); ``cu_q`` None: all of them."""
    if not q.is_cuda:
        _attention_reference(q[:rows], geo, cache, block_tables, cu_q, seq_lens, gate, gate_scale, out, scale)
        return
    H, G, D, B, dev, nb = geo.heads, geo.kv_heads, geo.dp, seq_lens.shape[0], q.device, cache.keys.shape[0]
    assert block_tables.stride(1) == 1 and out.stride(1) == 1 and (gate is None or (gate.dtype == torch.float32 and gate.stride(1) == 1))
    st, stream = ptr(status_tensor(dev)), stream_handle(dev)
    gate_args = (None, 0, ptr(gate), gate.stride(0) if gate is not None else 0, gate_scale)
    if q.dtype == torch.float32 or not geo.tensor_core:
        rc = _lib().rb_kv_simple(ptr(q), q.stride(0), ptr(cache.keys), ptr(cache.values), ptr(block_tables), ptr(cu_q), ptr(seq_lens), None, *gate_args,
                                 ptr(out), out.stride(0), H, G, D, block_tables.stride(0), nb, B, rows, max_q, geo.window, geo.chunk, _DT[q.dtype], scale,
                                 st, stream)
        check_rc(rc, "rb_kv_simple")
        return
    if cu_q is None:
        n_single = B
    if n_single > 0:
        rc = _lib().rb_kv_decode(ptr(q), q.stride(0), ptr(cache.keys), ptr(cache.values), ptr(block_tables), ptr(seq_lens), None, *gate_args, ptr(out),
                                 out.stride(0), ptr(workspace), n_single, H, G, D, block_tables.stride(0), nb, KV_BLOCK, splits, geo.window, geo.chunk,
                                 scale, st, stream)
        check_rc(rc, "rb_kv_decode", 2 if splits > 1 else 1)
    if n_single < B:
        rc = _flash_lib().rb_flash_fwd_ex(ptr(q), ptr(cache.keys), ptr(cache.values), ptr(out), out.stride(0), None, ptr(cu_q[n_single:]), None,
                                          ptr(seq_lens[n_single:]), ptr(block_tables[n_single:]), B - n_single, rows, nb, H, G, D, q.stride(0), 0, 0,
                                          max_q, block_tables.stride(0), 1, geo.window, geo.chunk, 1, ptr(gate),
                                          gate.stride(0) if gate is not None else 0, gate_scale, scale, st, stream)
        check_rc(rc, "rb_flash_fwd_ex")

"""Latent attention (csrc/latent_sm100.cu) and its PyTorch twins.

Per token the cache keeps one row for all heads: the RMS-normalised latent ``c`` and one rotated key part
(``LatentGeometry`` has the padded layout). Head ``h`` attends with key ``(W_uk[h] c, rotated part)`` and value
``W_uv[h] c`` under a causal sliding window, with ``exp(sink_h)`` in the softmax denominator and a gate on its output.

``latent_attention`` works on the cached rows themselves (queries multiplied by ``W_uk[h]`` beforehand, the sum of
latents by ``W_uv[h]`` afterwards: ``head_gemm_absorb`` / ``head_gemm_expand``); ``flash.flash_latent_prefill`` runs long
prompt portions on keys and values multiplied out from gathered rows. Everything is bf16 with 32-bit scores, weights,
norms and angles on the serving path, and fp32 throughout in the exact mode.
"""

from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle
from .gemm import RbGemmArgs, EPI_STORE, _lib as _gemm_lib

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p
LATENT_BLOCK = 16
_DT = {torch.bfloat16: 0, torch.float32: 1}


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


@dataclass(frozen=True)
class LatentGeometry:
    """Padded sizes of one latent-attention layer. Padding channels are zero in the weights, the queries and the cache."""

    heads: int
    dim: int           # unrotated query/key channels per head
    rot_dim: int       # rotated channels
    rot_pairs: int     # pairs that turn (the remaining rotated-part channels pass through)
    vdim: int
    kv_rank: int
    q_rank: int

    @property
    def dp(self) -> int:           # unrotated part of a head's query
        return _up(self.dim, 64)

    @property
    def rp(self) -> int:           # rotated part of a head's query
        return _up(self.rot_dim, 64)

    @property
    def vp(self) -> int:           # value channels of a head
        return _up(self.vdim, 64)

    @property
    def rw(self) -> int:           # latent columns of a cache row; the rotated part starts here
        return _up(self.kv_rank, 16)

    @property
    def cw(self) -> int:           # cache row
        return _up(self.rw + _up(self.rot_dim, 16), 32)

    @property
    def qp(self) -> int:           # query latent
        return _up(self.q_rank, 8)

    @property
    def proj(self) -> int:         # joint down projection: query latent | kv latent | rotated key part | gates
        return _up(self.q_rank + self.kv_rank + self.rot_dim + self.heads, 8)


def _lib() -> ctypes.CDLL:
    lib = _native.load("rb_latent")
    if not getattr(lib, "_rb_typed", False):
        lib.rb_latent_append.argtypes = ([c_vp, c_ll, c_vp, c_vp, c_float] + [c_vp] * 3 + [c_int, c_int, c_vp, c_ll, c_int, c_int, c_vp, c_ll, c_vp]
                                         + [c_int] * 6 + [c_vp, c_vp])
        lib.rb_latent_query.argtypes = [c_vp] * 3 + [c_int] * 3 + [c_vp, c_vp, c_ll] + [c_int] * 8 + [c_vp, c_vp]
        lib.rb_latent_attn.argtypes = [c_vp] * 11 + [c_ll] + [c_int] * 7 + [c_float] + [c_int] * 4 + [c_vp, c_vp]
        lib.rb_latent_plan.argtypes = [c_vp, c_vp] + [c_int] * 6 + [c_vp, c_vp]
        lib.rb_latent_gather.argtypes = [c_vp, c_vp] + [c_int] * 3 + [c_vp, c_vp, c_int, c_int, c_vp, c_vp] + [c_int] * 5 + [c_vp, c_vp]
        for f in ("rb_latent_append", "rb_latent_query", "rb_latent_attn", "rb_latent_plan", "rb_latent_gather"):
            getattr(lib, f).restype = c_int
        lib._rb_typed = True
    return lib


def _rotate_half_pairs(v: torch.Tensor, cs: torch.Tensor) -> torch.Tensor:
    """Rotate the first ``2 * pairs`` channels of ``v [T, ..., D]`` (fp32) by ``cs [T, pairs, 2]``."""
    n = cs.shape[1]
    shape = (cs.shape[0],) + (1,) * (v.dim() - 2) + (n,)
    c, s = cs[..., 0].reshape(shape), cs[..., 1].reshape(shape)
    a, b = v[..., :n], v[..., n:2 * n]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., 2 * n:]], -1)


# ------------------------------------------------------------------------------- norms, rotation, cache append
def latent_append(proj, geo: LatentGeometry, q_norm, kv_norm, eps: float, positions, slots, table, cache, cq, gate) -> None:
    """From the fp32 joint projection: normalised query latent -> ``cq``, normalised kv latent and rotated key part ->
    the cache rows at ``slots`` (negative: skipped), ``sigmoid`` of the gate logits -> ``gate [T, H]``."""
    T = proj.shape[0]
    q0, k0, r0 = geo.q_rank, geo.q_rank + geo.kv_rank, geo.q_rank + geo.kv_rank + geo.rot_dim
    if not proj.is_cuda:
        def rms(v, w):
            return v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w

        cq[:T, :q0] = rms(proj[:, :q0], q_norm).to(cq.dtype)
        gate[:T] = torch.sigmoid(proj[:, r0:r0 + geo.heads])
        ok = slots >= 0
        sl = slots[ok].long()
        flat = cache.view(-1, geo.cw)
        flat[sl, :geo.kv_rank] = rms(proj[ok][:, q0:k0], kv_norm).to(cache.dtype)
        flat[sl, geo.rw:geo.rw + geo.rot_dim] = _rotate_half_pairs(proj[ok][:, k0:r0], table[positions[ok].long()]).to(cache.dtype)
        return
    assert proj.dtype == torch.float32 and proj.stride(1) == 1 and cache.is_contiguous() and gate.dtype == torch.float32
    rc = _lib().rb_latent_append(ptr(proj), proj.stride(0), ptr(q_norm), ptr(kv_norm), eps, ptr(positions), ptr(slots), ptr(table),
                                 table.shape[0], geo.rot_pairs, ptr(cache), cache.shape[0] * LATENT_BLOCK, geo.cw, geo.rw, ptr(cq),
                                 cq.stride(0), ptr(gate), geo.q_rank, geo.kv_rank, geo.rot_dim, geo.heads, T, _DT[cq.dtype],
                                 ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_latent_append")


def latent_query(q, geo: LatentGeometry, positions, table, n_light: int, qn, qa) -> None:
    """Rotate the queries ``q [T, H, dp + rp]``. The first ``n_light`` tokens go head-major to ``qn [H, S, dp]`` (unrotated
    part) and ``qa [H, S, cw]`` (rotated part); the others are rotated in place."""
    T = q.shape[0]
    q3 = q.view(T, geo.heads, geo.dp + geo.rp)
    if not q.is_cuda:
        cs = table[positions.long().clamp(min=0)]
        rot = _rotate_half_pairs(q3[..., geo.dp:geo.dp + geo.rot_dim].float(), cs).to(q.dtype)
        qn[:, :n_light] = q3[:n_light, :, :geo.dp].transpose(0, 1)
        qa[:, :n_light, geo.rw:geo.rw + geo.rot_dim] = rot[:n_light].transpose(0, 1)
        q3[n_light:, :, geo.dp:geo.dp + geo.rot_dim] = rot[n_light:]
        return
    assert q.is_contiguous() and qn.is_contiguous() and qa.is_contiguous()
    rc = _lib().rb_latent_query(ptr(q), ptr(positions), ptr(table), table.shape[0], geo.rot_pairs, n_light, ptr(qn), ptr(qa), qa.shape[1],
                                geo.heads, geo.dp, geo.rp, geo.rot_dim, geo.cw, geo.rw, T, _DT[q.dtype],
                                ptr(status_tensor(q.device)), stream_handle(q.device))
    check_rc(rc, "rb_latent_query")


# ------------------------------------------------------------------------------- per-head products
_HEAD_TILES: dict[tuple, tuple[torch.Tensor, torch.Tensor, int]] = {}
_ROW_DST: dict[tuple, torch.Tensor] = {}


def _head_tiles(H: int, n: int, stride: int, N: int, b_step: int, bn: int, mode: int, device) -> tuple[torch.Tensor, torch.Tensor, int]:
    """Device tile table of ``H`` products over rows ``[h*stride, h*stride + n)``, cached."""
    key = (H, n, stride, N, b_step, bn, mode, device.index)
    if key not in _HEAD_TILES:
        if len(_HEAD_TILES) >= 4096:         # captured graphs keep theirs alive through live_tables()
            _HEAD_TILES.clear()
        # mode 0 names the tile's first B row, mode 1 the head's first B row (its tile column is n0)
        rows = [(h * stride + m, min(128, n - m), h * b_step + (n0 if mode == 0 else 0), n0) for h in range(H) for n0 in range(0, N, bn) for m in range(0, n, 128)]
        _HEAD_TILES[key] = (torch.tensor(rows, dtype=torch.int32).to(device), torch.tensor([len(rows)], dtype=torch.int32).to(device), len(rows))
    return _HEAD_TILES[key]


def live_tables() -> list:
    """The device tables made so far; whoever captured launches into a graph holds on to them."""
    return list(_HEAD_TILES.values()) + list(_ROW_DST.values())


def _head_bn(H: int, n: int, N: int, least: int) -> int:
    """Widest tile that still gives most SMs one: these products have a short K and many independent heads."""
    m_tiles = -(-n // 128)
    for bn in (256, 128, 64, 32):
        if bn >= least and (bn == least or (bn <= N and H * m_tiles * -(-N // bn) >= 120)):
            return bn
    return least


def _grouped(a, w, out, H, n, N, K, b_step, bn, mode, row_dst=None) -> None:
    table, count, tiles = _head_tiles(H, n, a.shape[1], N, b_step, bn, mode, a.device)
    args = RbGemmArgs()
    args.A[0], args.B[0], args.C = a.data_ptr(), w.data_ptr(), out.data_ptr()
    args.lda, args.ldb, args.ldc = a.stride(1), w.stride(0), out.stride(-2)
    args.M, args.N, args.K = a.shape[0] * a.shape[1], (N if mode == 1 else H * N), K
    args.a_parts = args.b_parts = 1
    args.b_mn_major = int(mode == 1)
    args.bn, args.epi_mode = bn, EPI_STORE
    args.rank, args.world = 0, 1
    args.tile_table, args.num_tiles_ptr = table.data_ptr(), count.data_ptr()
    args.group_n, args.max_tiles, args.max_ctas = N, tiles, min(tiles, 148)
    args.group_mode, args.group_b_rows = mode, w.shape[0] if mode == 1 else 0
    args.row_dst = row_dst.data_ptr() if row_dst is not None else None
    args.status = status_tensor(a.device).data_ptr()
    check_rc(_gemm_lib().rb_gemm_bf16_ex(ctypes.byref(args), stream_handle(a.device)), "rb_gemm_bf16_ex(heads)")


def head_gemm_absorb(a, w, out, n: int) -> None:
    """``out[h, t, :N] = a[h, t] @ w[h]`` for ``t < n``: ``a [H, S, K]``, ``w [H*K, N]``, ``out [H, S, >=N]``."""
    H, S, K = a.shape
    N = w.shape[1]
    if not a.is_cuda:
        out[:, :n, :N] = torch.einsum("htk,hkn->htn", a[:, :n].float(), w.view(H, K, N).float()).to(out.dtype)
        return
    if a.dtype == torch.float32:
        from .gemm import gemm_f32_batched

        gemm_f32_batched(a, w, out, n, N, K, H, (a.stride(1), w.stride(0), out.stride(1)), (a.stride(0), K * w.stride(0), out.stride(0)), b_kn=True)
        return
    assert K % 64 == 0
    _grouped(a, w, out, H, n, N, K, K, _head_bn(H, n, N, 64), 1)


def head_gemm_expand(a, w, out, n: int) -> None:
    """``out[t, h*N:(h+1)*N] = a[h, t] @ w[h].T`` for ``t < n``: ``a [H, S, K]``, ``w [H*N, K]``, ``out [T, H*N]``."""
    H, S, K = a.shape
    N = w.shape[0] // H
    if not a.is_cuda:
        out[:n] = torch.einsum("htk,hnk->thn", a[:, :n].float(), w.view(H, N, K).float()).reshape(n, H * N).to(out.dtype)
        return
    if a.dtype == torch.float32:
        from .gemm import gemm_f32_batched

        gemm_f32_batched(a, w, out, n, N, K, H, (a.stride(1), w.stride(0), out.stride(0)), (a.stride(0), N * w.stride(0), N))
        return
    key = (out.data_ptr(), H, S, N, out.stride(0), a.device.index)
    if key not in _ROW_DST:      # head-major rows land token-major: one destination address per (head, token)
        rows = min(S, out.shape[0])
        t = torch.arange(S, dtype=torch.int64).clamp(max=rows - 1)
        h = torch.arange(H, dtype=torch.int64)
        dst = out.data_ptr() + 2 * (t[None, :] * out.stride(0) + h[:, None] * N)
        _ROW_DST[key] = dst.reshape(-1).to(a.device)
    _grouped(a, w, out, H, n, N, K, N, _head_bn(H, n, N, 32), 0, _ROW_DST[key])


# ------------------------------------------------------------------------------- attention on the cached rows
def latent_units(B: int, heads: int, max_q: int) -> int:
    """Row tiles of a batch: 32 (token, head) rows each, or 16 where a sequence has no more."""
    rows = 32 if max_q * heads > 16 else 16
    return B * -(-max_q * heads // rows)


def latent_workspace(geos, device) -> torch.Tensor:
    """fp32 room for the partial results of units cut by a CTA boundary, for any batch of these geometries."""
    sms = torch.cuda.get_device_properties(device).multi_processor_count
    return torch.empty(2 * sms * 32 * (max(g.rw for g in geos) + 2), dtype=torch.float32, device=device)


def latent_plan(cu_q, seq_lens, geo: LatentGeometry, max_q: int, window: int, plan) -> None:
    """Prefix sums of the row tiles' key tiles -> ``plan [latent_units + 1]`` (int32): how ``latent_attention`` shares its
    work. One per batch, window and geometry; the CPU twin needs none."""
    if not seq_lens.is_cuda:
        return
    B = seq_lens.shape[0]
    assert plan.dtype == torch.int32 and plan.numel() >= latent_units(B, geo.heads, max_q) + 1
    check_rc(_lib().rb_latent_plan(ptr(cu_q), ptr(seq_lens), B, geo.heads, max_q, window, geo.cw, geo.rw, ptr(plan), stream_handle(seq_lens.device)), "rb_latent_plan")


def latent_attention(qa, cache, geo: LatentGeometry, block_tables, cu_q, seq_lens, sink, gate, out, *, scale: float, window: int,
                     rows: int, max_q: int, plan=None, workspace=None) -> None:
    """``out[h, t] = gate[t, h] * sum_j p_j c_j`` for the first ``rows`` tokens of ``qa [H, S, cw]``.

    ``cu_q`` ``[B+1]`` gives the rows of every sequence (None: one row per sequence); the new tokens are the last of the
    sequence's ``seq_lens`` keys and already in the cache. bf16 on the GPU needs the batch's ``plan`` and a
    ``latent_workspace``."""
    B = seq_lens.shape[0]
    H, S = qa.shape[0], qa.shape[1]
    if not qa.is_cuda:
        flat = cache.view(-1, geo.cw)
        for b in range(B):
            t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
            L = int(seq_lens[b])
            if L == 0 or t1 == t0:
                out[:, t0:t1] = 0
                continue
            pos = torch.arange(L - (t1 - t0), L)
            key = torch.arange(L)
            kv = flat[block_tables[b, key // LATENT_BLOCK].long() * LATENT_BLOCK + key % LATENT_BLOCK].float()
            s = torch.einsum("htc,kc->htk", qa[:, t0:t1].float(), kv) * scale
            dead = (key[None] > pos[:, None]) | (key[None] <= pos[:, None] - window)
            s = s.masked_fill(dead[None], -math.inf)
            full = torch.cat([s, sink.view(H, 1, 1).expand(H, t1 - t0, 1)], -1).softmax(-1)
            o = torch.einsum("htk,kc->htc", full[..., :-1], kv[:, :geo.rw]) * gate[t0:t1].T[..., None]
            out[:, t0:t1, :geo.rw] = o.to(out.dtype)
        return
    dt = _DT[qa.dtype]
    part_ml = None
    if dt == 0:
        n = workspace.numel() // (geo.rw + 2) * geo.rw
        part_ml = workspace[n:]
    assert qa.is_contiguous() and out.is_contiguous() and cache.is_contiguous() and sink.dtype == gate.dtype == torch.float32
    rc = _lib().rb_latent_attn(ptr(qa), ptr(cache), ptr(block_tables), ptr(cu_q), ptr(seq_lens), ptr(sink), ptr(gate), ptr(out), ptr(plan),
                               ptr(workspace), ptr(part_ml), S, H, geo.cw, geo.rw, out.shape[2], block_tables.stride(0),
                               cache.shape[0], window, scale, B, rows, max_q, dt, ptr(status_tensor(qa.device)), stream_handle(qa.device))
    check_rc(rc, "rb_latent_attn", 2 if dt == 0 else 1)


def latent_gather(cache, geo: LatentGeometry, block_tables, bt_row0: int, cu_k, k_lo, n_rows: int, lat, rot) -> None:
    """Pack the cached rows ``[k_lo[b], k_lo[b] + cu_k[b+1] - cu_k[b])`` of the sequences in ``block_tables[bt_row0:]``:
    latents -> ``lat [n, rw]``, rotated parts -> ``rot [n, rp]``."""
    B = k_lo.shape[0]
    if not cache.is_cuda:
        flat = cache.view(-1, geo.cw)
        for b in range(B):
            s, e = int(cu_k[b]), int(cu_k[b + 1])
            key = torch.arange(e - s) + int(k_lo[b])
            rows = flat[block_tables[bt_row0 + b, key // LATENT_BLOCK].long() * LATENT_BLOCK + key % LATENT_BLOCK]
            lat[s:e] = rows[:, :geo.rw]
            rot[s:e] = 0
            rot[s:e, :geo.rot_dim] = rows[:, geo.rw:geo.rw + geo.rot_dim]
        return
    rc = _lib().rb_latent_gather(ptr(cache), ptr(block_tables), bt_row0, block_tables.stride(0), cache.shape[0], ptr(cu_k), ptr(k_lo), B,
                                 n_rows, ptr(lat), ptr(rot), geo.cw, geo.rw, geo.rp, geo.rw, _up(geo.rot_dim, 16),
                                 ptr(status_tensor(cache.device)), stream_handle(cache.device))
    check_rc(rc, "rb_latent_gather")

"""RMSNorm, RoPE + paged KV append, SwiGLU, embedding (csrc/ops_sm100.cu) with reference twins.

The reference twins follow the rounding points of the bf16 Hugging Face modules, which are
also what the functional oracles in the reference implement
(rollouts/tools/functional_extractor/qwen_functional.py:46-150, 251-274).
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p


def _lib() -> ctypes.CDLL:
    lib = _native.load("rb_ops")
    if not getattr(lib, "_rb_typed", False):
        lib.rb_rmsnorm.argtypes = [c_vp, c_vp, c_vp, c_ll, c_int, c_ll, c_ll, c_float, c_vp]
        lib.rb_rope_kv_append.argtypes = [c_vp] * 9 + [c_float, c_int, c_int, c_int, c_int, c_int, c_ll, c_int, c_vp, c_vp]
        lib.rb_swiglu.argtypes = [c_vp, c_vp, c_ll, c_int, c_vp]
        lib.rb_swiglu_bwd.argtypes = [c_vp, c_vp, c_vp, c_ll, c_int, c_vp]
        lib.rb_swiglu_bounded.argtypes = [c_vp, c_vp, c_ll, c_int, c_vp, c_vp]
        lib.rb_swiglu_bounded.restype = c_int
        lib.rb_embedding.argtypes = [c_vp, c_vp, c_vp, c_int, c_int, c_int, c_vp, c_vp]
        lib.rb_transpose_bf16.argtypes = [c_vp, c_vp, c_int, c_int, c_vp]
        lib.rb_layernorm.argtypes = [c_vp, c_ll, c_vp, c_ll] + [c_vp] * 4 + [c_ll, c_int, c_int, c_int, c_float, c_int, c_vp, c_vp]
        lib.rb_clamped_glu.argtypes = [c_vp, c_vp, c_int, c_ll, c_int, c_float, c_vp]
        lib.rb_softcap.argtypes = [c_vp, c_ll, c_float, c_vp]
        lib.rb_stream_embed.argtypes = [c_vp, c_vp, c_ll, c_vp, c_ll, c_vp, c_ll, c_vp, c_ll] + [c_int] * 4 + [c_vp, c_vp]
        lib.rb_stream_norm.argtypes = ([c_vp, c_ll, c_vp, c_vp, c_ll, c_vp, c_vp, c_ll, c_int, c_vp, c_ll, c_vp, c_float, c_vp, c_ll, c_vp, c_ll, c_vp,
                                        c_vp] + [c_int] * 5 + [c_float, c_vp, c_vp])
        lib.rb_token_side.argtypes = [c_vp, c_ll, c_vp, c_vp, c_ll, c_int, c_vp, c_ll] + [c_int] * 4 + [c_vp, c_vp]
        lib.rb_stream_sandwich.argtypes = [ctypes.POINTER(SandwichArgs), c_vp]
        lib.rb_poly_norm.argtypes = [c_vp, c_ll, c_vp, c_vp, c_ll, c_int, c_int, c_int, c_float, c_int, c_vp]
        for f in ("rb_stream_sandwich", "rb_poly_norm", "rb_token_side", "rb_stream_embed", "rb_stream_norm", "rb_layernorm", "rb_clamped_glu", "rb_softcap", "rb_rmsnorm", "rb_rope_kv_append", "rb_swiglu", "rb_swiglu_bwd", "rb_embedding", "rb_transpose_bf16"):
            getattr(lib, f).restype = c_int
        lib._rb_typed = True
    return lib


# ------------------------------------------------------------------------------- RMSNorm
def rmsnorm_reference(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    xf = x.float()
    var = xf.pow(2).mean(-1, keepdim=True)
    y = (xf * torch.rsqrt(var + eps)).to(x.dtype)
    return w * y


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float = 1e-6, out: torch.Tensor | None = None) -> torch.Tensor:
    """Row RMSNorm over the last dim; also used per head (QK-norm) with ``x`` reshaped."""
    if not x.is_cuda:
        res = rmsnorm_reference(x, w, eps)
        if out is not None:
            out.copy_(res)
            return out
        return res
    d = x.shape[-1]
    x2 = x.reshape(-1, d)
    assert x2.stride(1) == 1 and x.dtype == torch.bfloat16
    if out is None:
        out = torch.empty_like(x2)
    o2 = out.reshape(-1, d)
    rc = _lib().rb_rmsnorm(ptr(x2), ptr(w), ptr(o2), x2.shape[0], d, x2.stride(0), o2.stride(0), eps, stream_handle(x.device))
    check_rc(rc, "rb_rmsnorm")
    return out.reshape(x.shape)


# ------------------------------------------------------------------------------- RoPE tables
def rope_table(max_pos: int, head_dim: int, theta: float, device=None, exact: bool = False) -> torch.Tensor:
    """``[max_pos, head_dim/2, 2]`` fp32 table of (cos, sin), HF ``inv_freq`` convention. ``exact`` forms the angles in
    float64 first, so that the table is right to fp32 at every position."""
    if exact:
        freq = float(theta) ** (-torch.arange(0, head_dim, 2, dtype=torch.float64) / max(head_dim, 1))
        ang = torch.outer(torch.arange(max_pos, dtype=torch.float64), freq)
        tab = torch.stack([ang.cos(), ang.sin()], dim=-1).float().contiguous()
        return tab.to(device) if device is not None else tab
    inv_freq = 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=torch.float32) / head_dim))
    pos = torch.arange(max_pos, dtype=torch.float32)
    ang = torch.outer(pos, inv_freq)
    tab = torch.stack([ang.cos(), ang.sin()], dim=-1).contiguous()
    return tab.to(device) if device is not None else tab


def frequency_table(max_pos: int, frequencies: list[float], amplitude: float = 1.0, device=None) -> torch.Tensor:
    """``[max_pos, n, 2]`` fp32 table of ``amplitude`` times (cos, sin) of position times frequency, angles formed in float64."""
    ang = torch.outer(torch.arange(max_pos, dtype=torch.float64), torch.tensor(frequencies, dtype=torch.float64))
    return (amplitude * torch.stack([ang.cos(), ang.sin()], dim=-1)).float().contiguous().to(device or "cpu")


def _rotate_reference(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    # x [T, H, D]; cos/sin [T, D/2] fp32 -> HF: cat(freqs,freqs), cast to x.dtype, x*cos + rotate_half(x)*sin
    c = torch.cat([cos, cos], -1).to(x.dtype)[:, None, :]
    s = torch.cat([sin, sin], -1).to(x.dtype)[:, None, :]
    half = x.shape[-1] // 2
    rot = torch.cat([-x[..., half:], x[..., :half]], -1)
    return x * c + rot * s


def rope_kv_append_reference(qkv, positions, slots, table, k_cache, v_cache, Hq, Hkv, D, q_norm_w=None, k_norm_w=None, eps=1e-6):
    T = qkv.shape[0]
    q, k, v = qkv.split([Hq * D, Hkv * D, Hkv * D], dim=-1)
    q = q.reshape(T, Hq, D)
    k = k.reshape(T, Hkv, D)
    v = v.reshape(T, Hkv, D)
    if q_norm_w is not None:
        q = rmsnorm_reference(q, q_norm_w, eps)
        k = rmsnorm_reference(k, k_norm_w, eps)
    cs = table[positions.long().clamp(min=0)]
    q = _rotate_reference(q, cs[..., 0], cs[..., 1])
    k = _rotate_reference(k, cs[..., 0], cs[..., 1])
    bs = k_cache.shape[2]
    ok = slots >= 0
    sl = slots[ok].long()
    k_cache[sl // bs, :, sl % bs] = k[ok]
    v_cache[sl // bs, :, sl % bs] = v[ok]
    return q.reshape(T, Hq * D)


def rope_kv_append(qkv, positions, slots, table, k_cache, v_cache, Hq, Hkv, D, q_norm_w=None, k_norm_w=None,
                   eps: float = 1e-6, q_out: torch.Tensor | None = None) -> torch.Tensor:
    """Rotate q and k, write k/v into the paged cache at ``slots``, return rotated q ``[T, Hq*D]``.

    ``k_cache``/``v_cache``: ``[num_blocks, Hkv, block_size, D]``; ``slots`` < 0 rows are skipped.
    """
    if not qkv.is_cuda:
        res = rope_kv_append_reference(qkv, positions, slots, table, k_cache, v_cache, Hq, Hkv, D, q_norm_w, k_norm_w, eps)
        if q_out is not None:
            q_out.copy_(res)
            return q_out
        return res
    T = qkv.shape[0]
    assert qkv.is_contiguous() and qkv.shape[1] == (Hq + 2 * Hkv) * D
    assert positions.dtype == torch.int32 and slots.dtype == torch.int32
    assert table.dtype == torch.float32 and table.is_contiguous()
    if q_out is None:
        q_out = torch.empty(T, Hq * D, dtype=qkv.dtype, device=qkv.device)
    nb, _, bs, _ = k_cache.shape
    rc = _lib().rb_rope_kv_append(
        ptr(qkv), ptr(q_out), ptr(k_cache), ptr(v_cache), ptr(positions), ptr(slots), ptr(table), ptr(q_norm_w),
        ptr(k_norm_w), eps, T, Hq, Hkv, D, bs, nb * bs, table.shape[0], ptr(status_tensor(qkv.device)),
        stream_handle(qkv.device))
    check_rc(rc, "rb_rope_kv_append")
    return q_out


# ------------------------------------------------------------------------------- SwiGLU
def swiglu_reference(gu: torch.Tensor) -> torch.Tensor:
    g, u = gu.chunk(2, dim=-1)
    return torch.nn.functional.silu(g) * u


def swiglu(gu: torch.Tensor, out: torch.Tensor | None = None, rows_dev: torch.Tensor | None = None) -> torch.Tensor:
    """``silu(gate) * up`` for ``gu = [gate | up]`` of shape ``[T, 2F]``. ``rows_dev`` (an int32 element on the
    device) caps the number of rows processed at run time; rows beyond it are left untouched."""
    if not gu.is_cuda:
        res = swiglu_reference(gu)
        if out is not None:
            out.copy_(res)
            return out
        return res
    T, F2 = gu.reshape(-1, gu.shape[-1]).shape
    F = F2 // 2
    assert gu.is_contiguous()
    if out is None:
        out = torch.empty(*gu.shape[:-1], F, dtype=gu.dtype, device=gu.device)
    if rows_dev is not None:
        assert rows_dev.dtype == torch.int32 and rows_dev.is_cuda
        rc = _lib().rb_swiglu_bounded(ptr(gu), ptr(out), T, F, rows_dev.data_ptr(), stream_handle(gu.device))
    else:
        rc = _lib().rb_swiglu(ptr(gu), ptr(out), T, F, stream_handle(gu.device))
    check_rc(rc, "rb_swiglu")
    return out


def swiglu_backward(gu: torch.Tensor, dout: torch.Tensor) -> torch.Tensor:
    if not gu.is_cuda:
        g, u = gu.float().chunk(2, dim=-1)
        sig = torch.sigmoid(g)
        silu = g * sig
        dy = dout.float()
        return torch.cat([dy * u * (sig + silu * (1 - sig)), dy * silu], -1).to(gu.dtype)
    T, F2 = gu.reshape(-1, gu.shape[-1]).shape
    dgu = torch.empty_like(gu)
    rc = _lib().rb_swiglu_bwd(ptr(gu), ptr(dout.contiguous()), ptr(dgu), T, F2 // 2, stream_handle(gu.device))
    check_rc(rc, "rb_swiglu_bwd")
    return dgu


# ------------------------------------------------------------------------------- embedding
def embedding(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    if not table.is_cuda:
        res = table[ids.long()]
        if out is not None:
            out.copy_(res)
            return out
        return res
    assert ids.dtype == torch.int32 and ids.is_contiguous()
    T = ids.numel()
    d = table.shape[1]
    if out is None:
        out = torch.empty(T, d, dtype=table.dtype, device=table.device)
    rc = _lib().rb_embedding(ptr(ids), ptr(table), ptr(out), T, d, table.shape[0], ptr(status_tensor(table.device)),
                             stream_handle(table.device))
    check_rc(rc, "rb_embedding")
    return out


def transpose(x: torch.Tensor) -> torch.Tensor:
    if not x.is_cuda:
        return x.t().contiguous()
    assert x.dim() == 2 and x.is_contiguous() and x.dtype == torch.bfloat16
    out = torch.empty(x.shape[1], x.shape[0], dtype=x.dtype, device=x.device)
    rc = _lib().rb_transpose_bf16(ptr(x), ptr(out), x.shape[0], x.shape[1], stream_handle(x.device))
    check_rc(rc, "rb_transpose_bf16")
    return out


# ------------------------------------------------------------------------------- 32-bit residual stream
_ACT = {torch.bfloat16: 0, torch.float32: 1}


def stream_embed(ids: torch.Tensor, table: torch.Tensor, d: int, x: torch.Tensor, a: torch.Tensor | None = None,
                 b: torch.Tensor | None = None) -> None:
    """``x[t, :d] = table[ids[t]]`` in fp32 and the same row in ``a`` and ``b`` (activation type, any row stride)."""
    T = ids.numel()
    if not table.is_cuda:
        row = table[ids.long(), :d]
        for dst in (x, a, b):
            if dst is not None:
                dst[:T, :d] = row.to(dst.dtype)
        return
    assert ids.dtype == torch.int32 and ids.is_contiguous() and x.dtype == torch.float32
    rc = _lib().rb_stream_embed(ptr(ids), ptr(table), table.stride(0), ptr(x), x.stride(0), ptr(a), a.stride(0) if a is not None else 0, ptr(b),
                                b.stride(0) if b is not None else 0, _ACT[table.dtype], T, d, table.shape[0], ptr(status_tensor(table.device)),
                                stream_handle(table.device))
    check_rc(rc, "rb_stream_embed")


def stream_norm(x: torch.Tensor, d: int, *, y1=None, y2=None, experts=None, expert_weights=None, top: int = 0, side=None, side_weight=None,
                mult: float = 1.0, copy=None, weight=None, eps: float = 0.0, h=None, rows=None) -> None:
    """What happens to the fp32 stream ``x [n, dp]`` (``d`` channels and zero padding) between two layers, in one pass:
    ``x += mult (y1 + y2 + sum_j expert_weights[t, j] experts[t, j] + side / rms(side) * side_weight)`` (the terms that are given),
    ``copy = x`` and ``h = x / rms(x) * weight`` in the activation type. Without ``expert_weights`` the ``top`` results of a token
    are added as they are. With ``rows`` only ``h[i]`` of row ``rows[i]``."""
    n = rows.numel() if rows is not None else x.shape[0]
    if not x.is_cuda:
        src = x if rows is None else x[rows.long()]
        assert rows is None or (y1 is None and y2 is None and experts is None and side is None)
        for y in (y1, y2):
            if y is not None:
                x += mult * y[:n]
        if experts is not None:
            k = top if expert_weights is None else expert_weights.shape[1]
            e = experts[:n * k].view(n, k, -1).float()
            x += mult * (e if expert_weights is None else e * expert_weights[:n, :, None]).sum(1)
        if side is not None:
            x += mult * side[:n] * torch.rsqrt(side[:n].pow(2).sum(-1, keepdim=True) / d + eps) * side_weight
        if copy is not None:
            copy[:n] = x.to(copy.dtype)
        if h is not None:
            h[:n] = (src * torch.rsqrt(src.pow(2).sum(-1, keepdim=True) / d + eps) * weight).to(h.dtype)
        return
    act = next((t for t in (h, copy, experts) if t is not None), x)
    assert x.dtype == torch.float32 and x.stride(1) == 1 and (rows is None or rows.dtype == torch.int32)
    assert all(t is None or t.stride(-1) == 1 for t in (y1, y2, experts, copy, h)) and (y1 is None or y2 is None or y1.stride(0) == y2.stride(0))
    y = y1 if y1 is not None else y2
    k = top if expert_weights is None else expert_weights.shape[1]
    rc = _lib().rb_stream_norm(ptr(x), x.stride(0), ptr(y1), ptr(y2), y.stride(0) if y is not None else 0, ptr(experts), ptr(expert_weights),
                               experts.stride(0) if experts is not None else 0, k, ptr(side), side.stride(0) if side is not None else 0,
                               ptr(side_weight), mult, ptr(copy), copy.stride(0) if copy is not None else 0, ptr(h), h.stride(0) if h is not None else 0, ptr(weight),
                               ptr(rows), x.shape[0], _ACT[act.dtype], n, d, x.shape[1], eps, ptr(status_tensor(x.device)),
                               stream_handle(x.device))
    check_rc(rc, "rb_stream_norm")


class SandwichArgs(ctypes.Structure):
    _fields_ = ([(n, c_vp) for n in ("x", "y", "y2", "w", "w2", "gate", "e", "p", "idx", "pass_", "post_weight", "post_bias", "post_alpha", "pre_weight",
                                     "pre_bias", "pre_alpha", "copy", "h", "rows", "status")]
                + [(n, c_ll) for n in ("ldx", "ldy", "ld_gate", "lde", "ld_pass", "ldc", "ldh")]
                + [(n, c_int) for n in ("k", "experts", "num_src_rows", "n", "d", "dp", "bounded", "dtype")]
                + [("pair_scale", c_float), ("eps", c_float)])


@dataclass
class StreamNorm:
    """A norm of stream rows: RMS norm, or with ``alpha`` (a scalar) ``tanh(alpha x) * weight + bias``; fp32 on the device."""

    weight: torch.Tensor
    bias: torch.Tensor | None = None
    alpha: torch.Tensor | None = None

    def reference(self, x: torch.Tensor, d: int, eps: float) -> torch.Tensor:
        if self.alpha is not None:
            return torch.tanh(self.alpha * x) * self.weight + self.bias
        return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / d + eps) * self.weight


@dataclass
class ChosenExperts:
    """Results ``e [T * k, dp]`` of the chosen experts with weights ``p`` and choices ``idx [T, k]``; choices from ``experts`` on stand for the
    rows of ``input``."""

    e: torch.Tensor
    p: torch.Tensor
    idx: torch.Tensor
    experts: int
    input: torch.Tensor


def stream_sandwich(x: torch.Tensor, d: int, *, y=None, pair=None, gate=None, chosen: ChosenExperts | None = None, post: StreamNorm | None = None,
                    pre: StreamNorm | None = None, eps: float = 0.0, copy=None, h=None, rows=None) -> None:
    """What happens to the fp32 stream ``x [n, dp]`` around a sublayer with norms before and after it, in one pass: ``x += post(v)``,
    ``copy = x`` and ``h = pre(x)`` in the activation type, with the sublayer's output ``v``

    * ``y`` times ``sigmoid(gate [n, >= 1])`` (its first column), if there is one, plus the weighted ``chosen`` experts, or
    * half the sum of two mixers' ``y`` and ``pair[0]``, each divided by its root mean square, times ``pair[1]`` and ``pair[2]``.

    With ``rows`` only ``h[i]`` of row ``rows[i]``."""
    n = rows.numel() if rows is not None else x.shape[0]
    update = y is not None or chosen is not None
    assert not (update and rows is not None) and (pair is None or (gate is None and chosen is None))
    if not x.is_cuda:
        src = x if rows is None else x[rows.long()]
        if update:
            v = torch.zeros_like(x)
            if pair is not None:
                v = 0.5 * sum(StreamNorm(w).reference(t[:n], d, eps) for t, w in ((y, pair[1]), (pair[0], pair[2])))
            elif y is not None:
                v = y[:n] if gate is None else y[:n] * torch.sigmoid(gate[:n, :1])
            if chosen is not None:
                k = chosen.p.shape[1]
                plain = (chosen.idx[:n] >= chosen.experts)[..., None]
                rows_of = torch.where(plain, chosen.input[:n, None].float(), chosen.e[:n * k].view(n, k, -1).float())
                v = v + (chosen.p[:n, :, None] * rows_of).sum(1)
            x += post.reference(v, d, eps)
        if copy is not None:
            copy[:n] = x.to(copy.dtype)
        if h is not None:
            h[:n] = pre.reference(src, d, eps).to(h.dtype)
        return
    a = SandwichArgs()
    assert x.dtype == torch.float32 and x.stride(1) == 1 and (rows is None or rows.dtype == torch.int32)
    for name, t in (("x", x), ("y", y), ("gate", gate), ("copy", copy), ("h", h), ("rows", rows), ("status", status_tensor(x.device))):
        setattr(a, name, t.data_ptr() if t is not None else None)
    a.ldx, a.ldy, a.ld_gate = x.stride(0), y.stride(0) if y is not None else 0, gate.stride(0) if gate is not None else 0
    a.ldc, a.ldh = copy.stride(0) if copy is not None else 0, h.stride(0) if h is not None else 0
    if pair is not None:
        assert pair[0].stride(0) == y.stride(0)
        a.y2, a.w, a.w2, a.pair_scale = pair[0].data_ptr(), pair[1].data_ptr(), pair[2].data_ptr(), 0.5
    act = next((t for t in (h, copy) if t is not None), x)
    if chosen is not None:
        act = chosen.e
        assert chosen.e.dtype == chosen.input.dtype and chosen.idx.dtype == torch.int32 and chosen.idx.is_contiguous() and chosen.p.is_contiguous()
        a.e, a.p, a.idx, a.pass_ = chosen.e.data_ptr(), chosen.p.data_ptr(), chosen.idx.data_ptr(), chosen.input.data_ptr()
        a.lde, a.ld_pass, a.k, a.experts = chosen.e.stride(0), chosen.input.stride(0), chosen.p.shape[1], chosen.experts
    assert (h is None or h.dtype == act.dtype) and (copy is None or copy.dtype == act.dtype)
    for name, norm in (("post", post if update else None), ("pre", pre if h is not None else None)):
        if norm is not None:
            for part in ("weight", "bias", "alpha"):
                t = getattr(norm, part)
                setattr(a, f"{name}_{part}", t.data_ptr() if t is not None else None)
    a.num_src_rows, a.n, a.d, a.dp, a.dtype, a.eps = x.shape[0], n, d, x.shape[1], _ACT[act.dtype], eps
    a.bounded = int(any(m is not None and m.alpha is not None for m in (post, pre)))
    check_rc(_lib().rb_stream_sandwich(ctypes.byref(a), stream_handle(x.device)), "rb_stream_sandwich")


def poly_norm(z: torch.Tensor, act: torch.Tensor, n: int, eps: float, out: torch.Tensor) -> torch.Tensor:
    """``act[0] N(z) + act[1] N(z^2) + act[2] N(z^3) + act[3]`` on the first ``n`` columns of the rows (zero behind them), ``N`` the division by
    the root mean square over those columns; ``act`` in fp32."""
    T = z.shape[0]
    if not z.is_cuda:
        v = z[:, :n].float()
        terms = (a * p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps) for a, p in zip(act, (v, v ** 2, v ** 3)))
        out[:T].zero_()
        out[:T, :n] = (sum(terms) + act[3]).to(out.dtype)
        return out
    assert z.stride(1) == out.stride(1) == 1 and z.dtype == out.dtype and act.dtype == torch.float32
    check_rc(_lib().rb_poly_norm(ptr(z), z.stride(0), ptr(act), ptr(out), out.stride(0), T, n, z.shape[1], eps, _ACT[z.dtype], stream_handle(z.device)),
             "rb_poly_norm")
    return out


def token_side(z: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, col: int, out: torch.Tensor, n: int) -> None:
    """``out[t, :n] = gelu_tanh(z[t, :n]) * table[ids[t], col : col + n]``, ``z`` in fp32."""
    T = ids.numel()
    if not z.is_cuda:
        g = torch.nn.functional.gelu(z[:T, :n], approximate="tanh")
        out[:T, :n] = (g * table[ids.long(), col:col + n].float()).to(out.dtype)
        return
    assert z.dtype == torch.float32 and z.stride(1) == out.stride(1) == table.stride(1) == 1 and out.dtype == table.dtype and ids.is_contiguous()
    rc = _lib().rb_token_side(ptr(z), z.stride(0), ptr(ids), ptr(table), table.stride(0), col, ptr(out), out.stride(0), n, T, table.shape[0],
                              _ACT[out.dtype], ptr(status_tensor(z.device)), stream_handle(z.device))
    check_rc(rc, "rb_token_side")


def layernorm_reference(v: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = v.float() - v.float().mean(-1, keepdim=True)
    return c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * w + b


def layernorm_residual(y: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float, x: torch.Tensor, xb: torch.Tensor,
                       d: int | None = None) -> None:
    """``x += layer_norm(y) * w + b`` on the first ``d`` (default: all) channels of the fp32 stream, and ``xb`` = the new ``x`` in
    the activation type."""
    n, d = x.shape[0], x.shape[1] if d is None else d
    if not x.is_cuda:
        x[:, :d] += layernorm_reference(y[:n, :d], w[:d], b[:d], eps)
        xb[:n, :d] = x[:, :d].to(xb.dtype)
        return
    assert y.dtype == torch.float32 and y.stride(1) == 1 and x.stride(1) == 1 and w.dtype == b.dtype == torch.float32
    rc = _lib().rb_layernorm(ptr(y), y.stride(0), ptr(x), x.stride(0), None, ptr(w), ptr(b), ptr(xb), xb.stride(0), _ACT[xb.dtype], n, d, eps, n,
                             ptr(status_tensor(x.device)), stream_handle(x.device))
    check_rc(rc, "rb_layernorm")


def layernorm_rows(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float, out: torch.Tensor, rows: torch.Tensor | None = None,
                   d: int | None = None) -> None:
    """``out[i] = layer_norm(x[rows[i]]) * w + b`` over the first ``d`` (default: all) channels (``rows`` None: all rows in order)."""
    d = x.shape[1] if d is None else d
    n = rows.numel() if rows is not None else x.shape[0]
    if not x.is_cuda:
        src = x if rows is None else x[rows.long()]
        out[:n, :d] = layernorm_reference(src[:, :d], w[:d], b[:d], eps).to(out.dtype)
        return
    assert x.stride(1) == 1 and x.dtype == torch.float32 and (rows is None or rows.dtype == torch.int32)
    rc = _lib().rb_layernorm(None, 0, ptr(x), x.stride(0), ptr(rows), ptr(w), ptr(b), ptr(out), out.stride(0), _ACT[out.dtype], n, d, eps, x.shape[0],
                             ptr(status_tensor(x.device)), stream_handle(x.device))
    check_rc(rc, "rb_layernorm")


def clamped_glu_reference(gu: torch.Tensor, limit: float | None) -> torch.Tensor:
    g, u = gu.float().chunk(2, dim=-1)
    if limit is None:
        return torch.nn.functional.silu(g) * u
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def clamped_glu(gu: torch.Tensor, limit: float | None, out: torch.Tensor | None = None) -> torch.Tensor:
    """``g sigmoid(1.702 g) (u + 1)`` with ``g = min(gate, limit)``, ``u = clamp(up, +-limit)`` for ``gu = [gate | up] [T, 2F]``;
    without a limit ``silu(gate) * up``."""
    T, F2 = gu.shape
    if out is None:
        out = torch.empty(T, F2 // 2, dtype=gu.dtype, device=gu.device)
    if not gu.is_cuda:
        out.copy_(clamped_glu_reference(gu, limit))
        return out
    assert gu.is_contiguous() and out.is_contiguous()
    check_rc(_lib().rb_clamped_glu(ptr(gu), ptr(out), _ACT[gu.dtype], T, F2 // 2, limit or 0.0, stream_handle(gu.device)), "rb_clamped_glu")
    return out


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(x / cap)`` in place on fp32."""
    if not x.is_cuda:
        x.copy_(cap * torch.tanh(x / cap))
        return x
    assert x.dtype == torch.float32 and x.is_contiguous()
    check_rc(_lib().rb_softcap(ptr(x), x.numel(), cap, stream_handle(x.device)), "rb_softcap")
    return x

"""Recurrent mixers with a matrix state per head (csrc/recurrent_sm100.cu) and their PyTorch twins.

All kinds write ``k v^T`` into a state that decays and read it with ``q``::

    S_t = a_t S_(t-1) + b_t k_t v_t^T          o_t = S_t^T q_t

* lightning: ``a`` is a constant of the head, ``b = 1`` (queries, keys and values come through SiLU, applied by the projection);
* matrix memory (mLSTM): capped gate logits ``i``, ``f``; ``log a = logsigmoid(f)``, ``b = exp(i)``, held relative to a running
  maximum ``m`` (from 0) so that nothing overflows; a second state ``n`` takes ``k`` alone and divides the output by
  ``max(|n . q|, exp(-m)) + 1e-6``;
* time mixing (RWKV): ``a`` is a vector, ``exp(-exp(z_t + w0))`` per key channel, ``b = 1``; ``o_t`` reads the state in front of the
  token and the token's own ``k v^T`` times a bonus ``u`` per key channel. Its projections read mixes of a token with the one
  before (``token_shift``);
* forget mixing (HGRN2): ``a = f_t`` per key channel, ``f = low + (1 - low) sigmoid(z + bias)`` with a lower bound per channel, and the key is
  ``1 - f_t``;
* delta rule: the state decays by a number ``g_t`` per head and then takes ``beta_t k_t (v_t - S^T k_t)^T``. ``delta_rows`` makes what it reads:
  short convolutions and SiLU, the factors that make queries and keys unit vectors, ``log g = -exp(A) softplus(z + dt)`` and ``beta``.

A sequence owns a slot of the state; one whose first new token is at position 0 starts from zero whatever the slot holds.
The state, the decays, the gates and the outputs are fp32; queries, keys and values come in the activation type.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from ._util import check_rc, ptr, status_tensor, stream_handle
from .grouped import look_back, move_history

c_int, c_ll, c_float, c_vp = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, ctypes.c_void_p
_DT = {torch.bfloat16: 0, torch.float32: 1}
MAX_DIM = 512
CHUNK = 128                  # tokens the chunked form takes at a time
STATE_COLS = 32              # value channels of one state tile; every tile carries its own n and m


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


@dataclass(frozen=True)
class RecurrentGeometry:
    """Padded sizes of one recurrent layer and its activation. Padding channels are zero in the weights."""

    heads: int
    dim: int
    vdim: int
    silu: bool                   # q, k and v come through SiLU (the projection applies it)
    gated: bool                  # mLSTM gates and normaliser (otherwise a decay per head or key channel)
    form: str = ""               # "forget": keys follow from the decay (heads are padded alike for keys and values); "delta"
    groups: int = 0              # heads of queries and keys, each shared by as many value heads (0: one each)

    @property
    def kp(self) -> int:
        return _up(max(self.dim, self.vdim) if self.form == "forget" else self.dim, 64)

    @property
    def vp(self) -> int:
        return _up(max(self.dim, self.vdim) if self.form == "forget" else self.vdim, 64)

    @property
    def key_heads(self) -> int:
        return self.groups or self.heads

    @property
    def q_scale(self) -> float:
        return self.dim ** -0.5 if self.gated or self.form == "delta" else 1.0

    @property
    def tiles(self) -> int:      # state tiles of a head
        return self.vp // STATE_COLS

    @property
    def proj(self) -> int:       # joint projection: q | k | v | output gate;  forget: q | v
        return self.offsets[3] + (0 if self.form == "forget" else self.heads * self.vp)

    @property
    def offsets(self) -> tuple[int, int, int, int]:
        a, b = self.key_heads * self.kp, self.heads * self.vp
        return (0, a, a, a + b) if self.form == "forget" else (0, a, 2 * a, 2 * a + b)

    @property
    def channels(self) -> int:           # of queries, keys and values
        return self.offsets[3]

    @property
    def silu_cols(self) -> int:          # columns of the joint projection that are activated
        return 0 if not self.silu else self.offsets[1] if self.form == "forget" else self.offsets[3]

    @property
    def state_floats(self) -> int:       # one sequence
        return self.heads * self.tiles * (self.kp * (STATE_COLS + 1) + 1)


@dataclass
class RecurrentState:
    """State of every slot: ``s [slots, H, tiles, kp, 32]``, ``n [slots, H, tiles, kp]``, ``m [slots, H, tiles]``."""

    s: torch.Tensor
    n: torch.Tensor
    m: torch.Tensor

    @staticmethod
    def zeros(geo: RecurrentGeometry, slots: int, device) -> "RecurrentState":
        lead = (slots, geo.heads, geo.tiles)
        return RecurrentState(*(torch.zeros(*lead, *tail, dtype=torch.float32, device=device) for tail in ((geo.kp, STATE_COLS), (geo.kp,), ())))


@dataclass
class TimeMix:
    """What time mixing adds to a recurrence: ``z [T, H*kp]`` fp32 with the decay ``exp(-exp(z + w0))``, the bonus of the current token."""

    z: torch.Tensor
    w0: torch.Tensor             # [H*kp]
    bonus: torch.Tensor          # [H*kp]


@dataclass
class ForgetMix:
    """Forget mixing: ``z [T, H*kp]`` fp32 with ``f = lower + (1 - lower) sigmoid(z + bias)``; ``keys [>= T, 2 H*kp]`` is room for the
    chunked form."""

    z: torch.Tensor
    bias: torch.Tensor           # [H*kp]
    lower: torch.Tensor          # [H*kp]
    keys: torch.Tensor | None = None

    w0 = property(lambda self: self.bias)
    bonus = property(lambda self: self.lower)


@dataclass
class DeltaRule:
    """What the delta rule reads besides its rows, fp32: ``units [T, 2G]`` factors of queries and keys, ``steps [T, 2H]`` logarithm of the decay
    and step size."""

    units: torch.Tensor
    steps: torch.Tensor


FORMS = {type(None): 0, TimeMix: 1, ForgetMix: 2, DeltaRule: 3}


def _lib() -> ctypes.CDLL:
    lib = _native.load("rb_recurrent")
    if not getattr(lib, "_rb_typed", False):
        lib.rb_recurrent_scan.argtypes = ([c_vp, c_ll] + [c_int] * 3 + [c_vp, c_ll] + [c_vp] * 3 + [c_float, c_float] + [c_vp] * 6
                                          + [c_vp, c_ll] + [c_int] * 8 + [c_vp, c_ll, c_vp, c_vp, c_int, c_int, c_vp, c_vp, c_int, c_vp, c_vp])
        lib.rb_delta_rows.argtypes = ([c_vp, c_ll, c_vp, c_int] + [c_vp] * 4 + [c_int, c_int, c_vp, c_ll, c_vp, c_ll] + [c_vp] * 4 + [c_int] * 6
                                      + [c_vp, c_vp])
        lib.rb_delta_chunks.argtypes = ([c_vp, c_ll, c_int, c_int, c_vp, c_vp, c_float] + [c_vp] * 7 + [c_ll, c_vp] + [c_int] * 8
                                        + [c_vp, c_vp])
        lib.rb_delta_workspace.argtypes, lib.rb_delta_workspace.restype = [c_int] * 4, c_ll
        lib.rb_token_shift.argtypes = [c_vp, c_ll, c_vp, c_int, c_vp, c_ll, c_ll, c_vp, c_vp, c_vp, c_vp] + [c_int] * 5 + [c_vp, c_vp]
        lib.rb_tanh_parts.argtypes = [c_vp, c_int, c_vp, c_vp, c_int, c_vp]
        lib.rb_recurrent_chunks.argtypes = ([c_vp, c_ll] + [c_int] * 3 + [c_vp, c_ll] + [c_vp] * 3 + [c_float, c_float] + [c_vp] * 9 + [c_ll, c_vp]
                                            + [c_int] * 8 + [c_vp, c_vp])
        lib.rb_recurrent_chunk_workspace.argtypes, lib.rb_recurrent_chunk_workspace.restype = [c_int] * 4, c_ll
        lib.rb_time_mix_chunks.argtypes = ([c_vp, c_ll] + [c_int] * 3 + [c_vp, c_ll] + [c_vp] * 9 + [c_float, c_vp, c_ll, c_vp, c_vp, c_ll] + [c_int] * 7
                                           + [c_vp, c_vp])
        lib.rb_time_mix_decode.argtypes = ([c_vp, c_ll] + [c_int] * 3 + [c_vp, c_ll] + [c_vp] * 3 + [c_float] + [c_vp] * 4 + [c_ll] + [c_int] * 7
                                           + [c_vp, c_vp])
        lib.rb_time_mix_workspace.argtypes, lib.rb_time_mix_workspace.restype = [c_int] * 3, c_ll
        lib.rb_gated_norm.argtypes = [c_vp, c_ll, c_vp, c_vp, c_ll, c_vp, c_ll] + [c_int] * 7 + [c_float, c_vp]
        for f in ("rb_recurrent_scan", "rb_recurrent_chunks", "rb_gated_norm", "rb_token_shift", "rb_tanh_parts", "rb_time_mix_chunks", "rb_time_mix_decode", "rb_delta_rows",
                  "rb_delta_chunks"):
            getattr(lib, f).restype = c_int
        lib._rb_typed = True
    return lib


def capped_gates(small, bias_i, bias_f, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """Logarithms of input and forget gate from ``small [T, i | f]``."""
    H = bias_i.shape[0]
    i = cap * torch.tanh((small[:, :H] + bias_i) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((small[:, H:2 * H] + bias_f) / cap))
    return i, f


def _split(proj, geo: RecurrentGeometry):
    T, (oq, ok, ov, og) = proj.shape[0], geo.offsets
    q, k = (proj[:, a:a + ok].float().reshape(T, geo.key_heads, -1) for a in (oq, ok))
    return q * geo.q_scale, k, proj[:, ov:og].float().reshape(T, geo.heads, -1)


def forget_gate(mix: ForgetMix, rows: int) -> torch.Tensor:
    return mix.lower + (1 - mix.lower) * torch.sigmoid(mix.z[:rows] + mix.bias)


def recurrent_scan(proj, small, geo: RecurrentGeometry, decay, bias_i, bias_f, cap: float, state: RecurrentState, slots, cu_q, seq_lens,
                   out, rows: int, n_seq: int, first: int = 0, mix: TimeMix | ForgetMix | DeltaRule | None = None) -> None:
    """Token-by-token form for the sequences ``first .. n_seq - 1`` (the last one ends at packed row ``rows``): ``out [T, H*vp]``
    fp32, state updated.

    ``proj [T, q | k | v | gate]``, ``small [T, i | f]`` fp32 (gated kinds), ``slots [B]`` (negative: padding), ``cu_q``
    ``[B+1]`` (None: one row per sequence), ``seq_lens [B]`` with the new tokens; ``mix`` for the other forms (the delta rule reads
    ``delta_rows``'s rows)."""
    H, KP, VP = geo.heads, geo.kp, geo.vp
    if not proj.is_cuda:
        q, k, v = _split(proj[:rows], geo)
        if isinstance(mix, TimeMix):
            keep = torch.exp(-torch.exp(mix.z[:rows] + mix.w0)).view(-1, H, KP)
            bonus = mix.bonus.view(H, KP, 1)
        elif isinstance(mix, ForgetMix):
            keep = forget_gate(mix, rows).view(-1, H, KP)
        elif isinstance(mix, DeltaRule):
            G = geo.key_heads
            q, k = (t.repeat_interleave(H // G, 1) for t in (q * mix.units[:rows, :G, None], k * mix.units[:rows, G:, None]))
            keep, beta = torch.exp(mix.steps[:rows, :H]), mix.steps[:rows, H:]
        if geo.gated:
            gi, gf = capped_gates(small[:rows], bias_i, bias_f, cap)
        for b in range(first, n_seq):
            t0, t1 = (b, b + 1) if cu_q is None else (int(cu_q[b]), int(cu_q[b + 1]))
            slot = int(slots[b])
            if slot < 0:
                out[t0:t1] = 0
                continue
            if int(seq_lens[b]) == t1 - t0:
                state.s[slot], state.n[slot], state.m[slot] = 0, 0, 0
            S = state.s[slot].permute(0, 2, 1, 3).reshape(H, KP, VP)
            n, m = state.n[slot, :, 0], state.m[slot, :, 0]
            for t in range(t0, t1):
                if isinstance(mix, ForgetMix):
                    S = keep[t][:, :, None] * S + (1 - keep[t])[:, :, None] * v[t][:, None, :]
                    out[t] = torch.einsum("hkv,hk->hv", S, q[t]).reshape(-1)
                    continue
                if isinstance(mix, DeltaRule):
                    S = keep[t][:, None, None] * S
                    u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
                    S = S + k[t][:, :, None] * u[:, None, :]
                    out[t] = torch.einsum("hkv,hk->hv", S, q[t]).reshape(-1)
                    continue
                if mix is not None:
                    kv = k[t][:, :, None] * v[t][:, None, :]
                    out[t] = torch.einsum("hkv,hk->hv", S + bonus * kv, q[t]).reshape(-1)
                    S = keep[t][:, :, None] * S + kv
                    continue
                if geo.gated:
                    new = torch.maximum(gf[t] + m, gi[t])
                    a, w = torch.exp(gf[t] + m - new), torch.exp(gi[t] - new)
                    m = new
                else:
                    a, w = decay, torch.ones_like(decay)
                kw = k[t] * w[:, None]
                S = a[:, None, None] * S + kw[:, :, None] * v[t][:, None, :]
                o = torch.einsum("hkv,hk->hv", S, q[t])
                if geo.gated:
                    n = a[:, None] * n + kw
                    o = o / (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6)[:, None]
                out[t] = o.reshape(-1)
            state.s[slot] = S.view(H, KP, geo.tiles, STATE_COLS).permute(0, 2, 1, 3)
            state.n[slot], state.m[slot] = n[:, None], m[:, None]
        return
    oq, ok, ov, _ = geo.offsets
    assert proj.stride(1) == 1 and out.dtype == torch.float32 and out.stride(1) == 1 and (cu_q is not None or first == 0) and geo.kp <= MAX_DIM
    vectors, delta = (mix if isinstance(mix, (TimeMix, ForgetMix)) else None), (mix if isinstance(mix, DeltaRule) else None)
    rc = _lib().rb_recurrent_scan(ptr(proj), proj.stride(0), oq, ok, ov, ptr(small), small.stride(0) if small is not None else 0, ptr(decay),
                                  ptr(bias_i), ptr(bias_f), cap, geo.q_scale, ptr(state.s), ptr(state.n), ptr(state.m),
                                  ptr(slots[first:]), ptr(cu_q[first:]) if cu_q is not None else None, ptr(seq_lens[first:]), ptr(out), out.stride(0), H, geo.dim, KP, VP,
                                  n_seq - first, state.s.shape[0],
                                  int(geo.gated), rows, ptr(vectors.z) if vectors is not None else None, vectors.z.stride(0) if vectors is not None else 0,
                                  ptr(vectors.w0) if vectors is not None else None, ptr(vectors.bonus) if vectors is not None else None, FORMS[type(mix)],
                                  H // geo.key_heads, ptr(delta.units) if delta is not None else None, ptr(delta.steps) if delta is not None else None,
                                  _DT[proj.dtype],
                                  ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_recurrent_scan")


@dataclass
class ChunkTable:
    """Device tables of the chunked form: ``chunks [n, 4]`` (first packed row, tokens, sequence, starts a portion) and
    ``seq_chunks [B + 1]`` for the packed sequences ``first ..`` of a batch."""

    chunks: torch.Tensor
    seq_chunks: torch.Tensor
    first: int

    @staticmethod
    def make(host_cu_q: list[int], first: int, device) -> "ChunkTable":
        rows, starts = [], [0]
        for i in range(first, len(host_cu_q) - 1):
            for t in range(host_cu_q[i], host_cu_q[i + 1], CHUNK):
                rows.append((t, min(CHUNK, host_cu_q[i + 1] - t), i - first, int(t == host_cu_q[i])))
            starts.append(len(rows))
        flat = torch.tensor([x for r in rows for x in r] + starts, dtype=torch.int32).to(device)
        return ChunkTable(flat[:4 * len(rows)].view(-1, 4), flat[4 * len(rows):], first)


def chunked_supported(geo: RecurrentGeometry) -> bool:
    """Padded key sizes the tensor-core kernels are built for."""
    return geo.kp <= 256


def recurrent_chunks(proj, small, geo: RecurrentGeometry, decay, bias_i, bias_f, cap: float, state: RecurrentState, slots, cu_q, seq_lens, out,
                     table: ChunkTable, workspace) -> None:
    """The recurrence over the sequences of ``table`` in chunks of 128 tokens (bf16 activations on the GPU): rows
    ``cu_q[first] ..`` of ``out``, state updated. ``workspace``: ``chunk_workspace`` bytes."""
    _, ok, ov, _ = geo.offsets
    n, B, f = table.chunks.shape[0], table.seq_chunks.shape[0] - 1, table.first
    assert proj.is_cuda and proj.dtype == torch.bfloat16 and proj.stride(1) == out.stride(1) == 1 and out.dtype == torch.float32
    assert workspace.numel() * workspace.element_size() >= chunk_workspace(n, geo)
    rc = _lib().rb_recurrent_chunks(ptr(proj), proj.stride(0), 0, ok, ov, ptr(small), small.stride(0) if small is not None else 0, ptr(decay), ptr(bias_i),
                                    ptr(bias_f), cap, geo.q_scale, ptr(state.s), ptr(state.n), ptr(state.m),
                                    ptr(table.chunks), ptr(table.seq_chunks), ptr(slots[f:]), ptr(cu_q[f:]), ptr(seq_lens[f:]), ptr(out),
                                    out.stride(0), ptr(workspace), n, B, geo.heads, geo.dim, geo.kp, geo.vp, state.s.shape[0], int(geo.gated), ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_recurrent_chunks", 4)


def chunk_workspace(n_chunks: int, geo: RecurrentGeometry) -> int:
    return int(_lib().rb_recurrent_chunk_workspace(n_chunks, geo.heads, geo.kp, geo.vp))


def time_mix_decode(proj, geo: RecurrentGeometry, mix: TimeMix | ForgetMix, state: RecurrentState, slots, seq_lens, norm, eps: float, out,
                    n: int) -> None:
    """Time mixing of the first ``n`` sequences, one row each, norm per head and SiLU gate included (forget mixing: no gate): rows of ``out
    [>= n, H*vp]`` in the activation type, state updated."""
    _, ok, ov, og = geo.offsets
    forget = isinstance(mix, ForgetMix)
    if not proj.is_cuda or geo.kp != 64:
        o = torch.empty(n, geo.heads * geo.vp, dtype=torch.float32, device=proj.device)
        recurrent_scan(proj, None, geo, None, None, None, 1.0, state, slots, None, seq_lens, o, n, n, mix=mix)
        gated_norm(o, norm, None if forget else proj[:, og:], geo, eps, out, True, silu=True)
        return
    assert proj.stride(1) == out.stride(1) == 1 and proj.dtype == out.dtype and mix.z.dtype == norm.dtype == torch.float32
    rc = _lib().rb_time_mix_decode(ptr(proj), proj.stride(0), ok, ov, og, ptr(mix.z), mix.z.stride(0), ptr(mix.w0), ptr(mix.bonus), ptr(norm), eps,
                                   ptr(state.s), ptr(slots), ptr(seq_lens), ptr(out), out.stride(0), n, geo.heads, geo.dim, geo.vdim,
                                   state.s.shape[0], int(forget), _DT[proj.dtype], ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_time_mix_decode")


def time_mix_chunked_supported(geo: RecurrentGeometry) -> bool:
    return geo.kp in (64, 128) and geo.kp == geo.vp


def time_mix_chunks(proj, geo: RecurrentGeometry, mix: TimeMix | ForgetMix, state: RecurrentState, slots, cu_q, seq_lens, norm, eps: float, out, table: ChunkTable,
                    workspace) -> None:
    """Time mixing (forget mixing: without a gate) over the sequences of ``table`` in chunks of 128 tokens, norm per head and SiLU gate included
    (bf16 activations on the GPU): rows ``cu_q[first] ..`` of ``out [T, H*vp]``, state updated. Their rows of ``mix.z`` are overwritten."""
    _, ok, ov, og = geo.offsets
    n, B, f = table.chunks.shape[0], table.seq_chunks.shape[0] - 1, table.first
    assert proj.is_cuda and proj.dtype == out.dtype == torch.bfloat16 and proj.stride(1) == out.stride(1) == 1
    assert workspace.numel() * workspace.element_size() >= time_mix_workspace(n, geo)
    keys = mix.keys if isinstance(mix, ForgetMix) else None
    assert keys is None or (keys.dtype == torch.bfloat16 and keys.stride(1) == 1 and keys.shape[0] >= proj.shape[0])
    assert keys is not None or isinstance(mix, TimeMix)
    rc = _lib().rb_time_mix_chunks(ptr(proj), proj.stride(0), ok, ov, og, ptr(mix.z), mix.z.stride(0), ptr(mix.w0), ptr(mix.bonus), ptr(state.s),
                                   ptr(table.chunks), ptr(table.seq_chunks), ptr(slots[f:]), ptr(cu_q[f:]), ptr(seq_lens[f:]), ptr(norm), eps, ptr(out),
                                   out.stride(0), ptr(workspace), ptr(keys), keys.stride(0) if keys is not None else 0, n, B, geo.heads, geo.dim, geo.vdim,
                                   geo.kp, state.s.shape[0],
                                   ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_time_mix_chunks", 3)


def time_mix_workspace(n_chunks: int, geo: RecurrentGeometry) -> int:
    return int(_lib().rb_time_mix_workspace(n_chunks, geo.heads, geo.kp))


# ------------------------------------------------------------------------------- delta rule
MAX_TAPS = 16


def delta_rows(proj, small, geo: RecurrentGeometry, conv, history, cu_q, positions, state_slots, rate, dt_bias, rows, mix: DeltaRule) -> None:
    """From the joint projection ``proj [T, q | k | v | ..]`` and the logits ``small [T, step size | decay]`` (fp32): convolved and activated
    ``rows [>= T, q | k | v]`` and ``mix``'s factors, decays and step sizes. ``conv [taps, channels]`` fp32, latest tap last; ``history [slots,
    taps - 1, channels]`` (None: one tap) moves on; ``rate = exp(A_log)``, ``dt_bias [H]`` fp32."""
    T, H, G, C, taps = proj.shape[0], geo.heads, geo.key_heads, geo.channels, conv.shape[0]
    if not proj.is_cuda:
        u = proj[:, :C]
        x = u.float() * conv[-1]
        if taps > 1:
            back = look_back(u, taps - 1, history, cu_q, positions, state_slots).float()
            x = x + sum(conv[taps - 1 - d] * back[:, d - 1] for d in range(1, taps))
            move_history(u, history, cu_q, state_slots)
        rows[:T, :C] = torch.nn.functional.silu(x).to(rows.dtype)
        qk = rows[:T, :geo.offsets[2]].float().reshape(T, 2 * G, geo.kp)
        mix.units[:T] = torch.rsqrt(qk.pow(2).sum(-1) + 1e-6)
        mix.steps[:T, :H] = -rate * torch.nn.functional.softplus(small[:, H:2 * H] + dt_bias)
        mix.steps[:T, H:] = torch.sigmoid(small[:, :H])
        return
    assert proj.stride(1) == rows.stride(1) == small.stride(1) == 1 and proj.dtype == rows.dtype and small.dtype == torch.float32
    assert mix.units.is_contiguous() and mix.steps.is_contiguous() and mix.units.shape[1] == 2 * G and mix.steps.shape[1] == 2 * H and conv.is_contiguous()
    rc = _lib().rb_delta_rows(ptr(proj), proj.stride(0), ptr(conv), taps, ptr(history), ptr(cu_q), ptr(positions), ptr(state_slots),
                              T if cu_q is None else cu_q.numel() - 1, history.shape[0] if history is not None else 1 << 30, ptr(rows), rows.stride(0),
                              ptr(small), small.stride(0), ptr(rate), ptr(dt_bias), ptr(mix.units), ptr(mix.steps), G, H, geo.kp, geo.vp, T,
                              _DT[proj.dtype], ptr(status_tensor(proj.device)), stream_handle(proj.device))
    check_rc(rc, "rb_delta_rows", 2 if cu_q is not None and taps > 1 else 1)


def delta_chunked_supported(geo: RecurrentGeometry) -> bool:
    return geo.kp in (64, 128)


def delta_chunks(rows, geo: RecurrentGeometry, mix: DeltaRule, state: RecurrentState, slots, cu_q, seq_lens, out, table: ChunkTable,
                 workspace) -> None:
    """The delta rule over the sequences of ``table`` in chunks of 128 tokens (bf16 rows on the GPU): fp32 rows ``cu_q[first] ..`` of ``out``, state
    updated. ``workspace``: ``delta_workspace`` bytes."""
    _, ok, ov, _ = geo.offsets
    n, B, f = table.chunks.shape[0], table.seq_chunks.shape[0] - 1, table.first
    assert rows.is_cuda and rows.dtype == torch.bfloat16 and rows.stride(1) == out.stride(1) == 1
    assert out.dtype == torch.float32 and workspace.numel() * workspace.element_size() >= delta_workspace(n, geo)
    rc = _lib().rb_delta_chunks(ptr(rows), rows.stride(0), ok, ov, ptr(mix.units), ptr(mix.steps), geo.q_scale, ptr(state.s), ptr(table.chunks),
                                ptr(table.seq_chunks), ptr(slots[f:]), ptr(cu_q[f:]), ptr(seq_lens[f:]), ptr(out),
                                out.stride(0), ptr(workspace), n, B, geo.heads, geo.heads // geo.key_heads, geo.dim, geo.kp, geo.vp, state.s.shape[0],
                                ptr(status_tensor(rows.device)), stream_handle(rows.device))
    check_rc(rc, "rb_delta_chunks", 3)


def delta_workspace(n_chunks: int, geo: RecurrentGeometry) -> int:
    return int(_lib().rb_delta_workspace(n_chunks, geo.heads, geo.kp, geo.vp))


def token_shift(h, mu, out, history, cu_q, positions, state_slots) -> None:
    """``out[s, t] = h_t + (h_(t-1) - h_t) mu[s]`` for the packed rows ``h [T, w]``, ``mu [mixes, w]`` fp32, ``out [mixes, >= T, w]``. The token
    before a portion comes from ``history [slots, 1, w]`` (zeros before a sequence), which moves on."""
    T = h.shape[0]
    if not h.is_cuda:
        back = look_back(h, 1, history, cu_q, positions, state_slots)[:, 0].float()
        for s in range(mu.shape[0]):
            out[s, :T] = (h.float() + (back - h.float()) * mu[s]).to(out.dtype)
        move_history(h, history, cu_q, state_slots)
        return
    assert h.stride(1) == out.stride(2) == 1 and mu.is_contiguous() and history.is_contiguous() and mu.dtype == torch.float32
    rc = _lib().rb_token_shift(ptr(h), h.stride(0), ptr(mu), mu.shape[0], ptr(out), out.stride(0), out.stride(1), ptr(history), ptr(cu_q), ptr(positions),
                               ptr(state_slots), T if cu_q is None else cu_q.numel() - 1, history.shape[0], h.shape[1], T, _DT[h.dtype],
                               ptr(status_tensor(h.device)), stream_handle(h.device))
    check_rc(rc, "rb_token_shift", 1 if cu_q is None else 2)


def tanh_parts(x, out) -> None:
    """``tanh`` of contiguous fp32 rows ``x [T, n]`` as operand of an exact product: fp32 ``out [T, n]``, or bf16 ``out [T, 2n]`` with what
    the first ``n`` columns lack in the others."""
    T, n = x.shape
    assert out.shape[1] == (n if out.dtype == torch.float32 else 2 * n)
    if not x.is_cuda:
        v = torch.tanh(x)
        out[:T, :n] = v.to(out.dtype)
        if out.dtype != torch.float32:
            out[:T, n:] = (v - out[:T, :n].float()).to(out.dtype)
        return
    assert x.is_contiguous() and out.is_contiguous()
    f32 = out.dtype == torch.float32
    check_rc(_lib().rb_tanh_parts(ptr(x), n, None if f32 else ptr(out), ptr(out) if f32 else None, T, stream_handle(x.device)), "rb_tanh_parts")


def gated_norm(o, weight, gate, geo: RecurrentGeometry, eps: float, out, per_head: bool, silu: bool = False) -> None:
    """``out = o / rms(o) * weight * sigmoid(gate)`` (``silu``: times ``silu(gate)``; without a gate: as it is) on ``[T, H*vp]``; the mean square is taken over one
    head's ``vdim`` channels (``per_head``) or over all heads'."""
    T, H, VP = o.shape[0], geo.heads, geo.vp
    if not o.is_cuda:
        x = o.view(T, H, VP)
        ms = x.pow(2).sum(-1) / geo.vdim if per_head else (x.pow(2).sum((1, 2)) / (H * geo.vdim))[:, None].expand(T, H)
        y = x * torch.rsqrt(ms + eps)[..., None] * weight.view(1, H, VP)
        if gate is not None:
            y = y * (torch.nn.functional.silu if silu else torch.sigmoid)(gate[:T].float().reshape(T, H, VP))
        out[:T] = y.reshape(T, H * VP).to(out.dtype)
        return
    assert o.dtype == torch.float32 and o.stride(1) == out.stride(1) == 1 and (gate is None or (gate.stride(1) == 1 and gate.dtype == out.dtype))
    rc = _lib().rb_gated_norm(ptr(o), o.stride(0), ptr(weight), ptr(gate), gate.stride(0) if gate is not None else 0, ptr(out), out.stride(0), H, geo.vdim, VP, int(per_head),
                              int(silu), T, _DT[out.dtype], eps, stream_handle(o.device))
    check_rc(rc, "rb_gated_norm")

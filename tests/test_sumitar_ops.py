"""The operations behind the Sumitar design one by one against the plain oracle (``sumitar_oracle.py``): CPU twins, and on a GPU the
kernels in bf16 and fp32. Recurrences carry a token that late queries look for, convolutions dirty histories, routers corrections that
decide, so that a lost state, a wrong chunk border or a weight that took the correction in shows."""

import pytest
import sumitar_oracle as oracle
import torch
from test_recurrent_ops import PLACES, close, i32, padded, rand

from research_b200 import ops
from research_b200.ops.experts import ExpertsGeometry, ExpertsScratch, route_reference
from research_b200.ops.grouped import KV_BLOCK, GroupedCache, GroupedGeometry
from research_b200.ops.recurrent import (ChunkTable, DeltaRule, ForgetMix, RecurrentGeometry, RecurrentState, delta_chunked_supported, delta_workspace,
                                         time_mix_chunked_supported, time_mix_workspace)


def columns(x, p, dev):
    """[h, d] fp32 vectors of heads -> [h * p] on the device."""
    return padded(x[None], p).view(-1).to(dev)


class Batches:
    """Feeds sequences in portions: packs the new rows of a step as the engine does (single tokens, short portions, long ones)."""

    def __init__(self, lens, slots, dev):
        self.lens, self.slots, self.dev, self.done = lens, slots, dev, [0] * len(lens)

    def step(self, parts, chunks):
        order = sorted(parts, key=lambda b: parts[b])
        self.order, self.at = order, {b: (self.done[b], self.done[b] + parts[b]) for b in order}
        self.cu = [0]
        for b in order:
            self.cu.append(self.cu[-1] + parts[b])
            self.done[b] += parts[b]
        self.T = self.cu[-1]
        self.positions = torch.cat([torch.arange(*self.at[b]) for b in order]).int().to(self.dev)
        self.state_slots, self.cut = i32([self.slots[b] for b in order], self.dev), i32(self.cu, self.dev)
        self.seq_lens = i32([self.at[b][1] for b in order], self.dev)
        self.single = next((i for i, b in enumerate(order) if parts[b] > 1), len(order))
        self.short = next((i for i, b in enumerate(order) if parts[b] > 16), len(order)) if chunks else len(order)
        self.table = ChunkTable.make(self.cu, self.short, self.dev) if self.short < len(order) else None
        return self

    def rows(self, data):
        """[sum of new rows, ..] of per-sequence tensors."""
        return torch.cat([data[b][slice(*self.at[b])] for b in self.order])

    def split(self, out, got):
        for i, b in enumerate(self.order):
            got[b].append(out[self.cu[i]:self.cu[i + 1]].cpu())


LENS, SLOTS = [150, 60, 273, 9], [4, 0, 5, 2]
STEPS = ({0: 17, 1: 60, 2: 129}, {0: 2, 2: 1, 3: 1}, {0: 130, 2: 128, 3: 3}, {0: 1, 2: 2, 3: 5}, {2: 13})


# ------------------------------------------------------------------------------------------ forget mixing
def forget_case(heads, dim, vdim, n, seed):
    """q, v (rounded to bf16), logits and lower bounds; the second token is written into slow channels and found again by the last queries."""
    q, v = (rand(n, heads, c, seed=seed + i, dtype=torch.bfloat16) for i, c in enumerate((dim, vdim)))
    z = rand(n, heads, dim, seed=seed + 5) * 2
    slow = torch.arange(dim) % 3 == 0
    z[..., slow] = 8 + z[..., slow]
    if n > 3:
        v[1] *= 6
        z[1, :, slow] = -4
        q[n - 2:] = torch.where(slow, rand(heads, dim, seed=seed + 6).abs() * 2, 0.1).bfloat16()
    return q, v.bfloat16(), z


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", [(3, 24, 20), (1, 7, 50), (5, 64, 64), (2, 128, 128), (2, 30, 100), (3, 100, 40), (1, 200, 90)])
def test_forget_mixing_in_portions_slots_and_batches(place, shape):
    """Portions that straddle chunk borders, down to two tokens, then single tokens, in dirty slots: scan, decode kernel and chunks."""
    dev, dt = place
    H, D, E = shape
    geo = RecurrentGeometry(H, D, E, silu=True, gated=False, form="forget")
    eps, n = 1e-4, geo.heads * geo.kp
    bias, lower, norm = rand(H, D, seed=50) * 0.5, torch.rand(H, D, generator=torch.Generator().manual_seed(51)) * (torch.arange(D) % 2), rand(E, seed=52) + 1.5
    data = [forget_case(H, D, E, m, 10 * b + 100) for b, m in enumerate(LENS)]
    want = []
    for q, v, z in data:
        f = lower.double() + (1 - lower.double()) * torch.sigmoid(z.double() + bias.double())
        want.append(oracle.rms(oracle.forget_scan(q.double(), f, v.double()), eps) * norm.double())
    state = RecurrentState.zeros(geo, 6, dev)
    state.s.fill_(7.0)
    bias_p, lower_p, norm_p = columns(bias, geo.kp, dev), columns(lower, geo.kp, dev), columns(norm.expand(H, E), geo.vp, dev)
    got, bt = [[] for _ in LENS], Batches(LENS, SLOTS, dev)
    for parts in STEPS:
        b = bt.step(parts, dt == torch.bfloat16 and dev == "cuda" and time_mix_chunked_supported(geo))
        q, v, z = (b.rows([d[i] for d in data]) for i in range(3))
        proj = torch.cat([padded(q, geo.kp), padded(v, geo.vp), torch.full((b.T, 8), 9.0)], 1).to(dt).to(dev)
        mix = ForgetMix(padded(z, geo.kp).to(dev), bias_p, lower_p, torch.full((b.T, 2 * n), 3.0, dtype=dt, device=dev))
        o, out = torch.full((b.T, H * geo.vp), 9.0, device=dev), torch.full((b.T, H * geo.vp + 8), 9.0, dtype=dt, device=dev)[:, :H * geo.vp]
        if b.single:
            ops.time_mix_decode(proj, geo, mix, state, b.state_slots, b.seq_lens, norm_p, eps, out, b.single)
        if b.short > b.single:
            ops.recurrent_scan(proj, None, geo, None, None, None, 1.0, state, b.state_slots, b.cut, b.seq_lens, o, b.cu[b.short], b.short, b.single, mix=mix)
            ops.gated_norm(o[b.single:b.cu[b.short]], norm_p, None, geo, eps, out[b.single:], True)
        if b.table is not None:
            room = torch.empty(time_mix_workspace(b.table.chunks.shape[0], geo), dtype=torch.uint8, device=dev)
            ops.time_mix_chunks(proj, geo, mix, state, b.state_slots, b.cut, b.seq_lens, norm_p, eps, out, b.table, room)
        b.split(out, got)
    for i, m in enumerate(LENS):
        o = torch.cat(got[i]).view(m, H, geo.vp)
        assert geo.vp == E or o[..., E:].abs().max() == 0
        close(o[..., :E], want[i], dt, (shape, i))
    for part in (1, 3):         # slots nobody owns keep what they held
        assert (state.s[part] == 7.0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,E,B", [(6, 40, 64, 300), (32, 64, 50, 64), (1, 64, 64, 1), (3, 128, 70, 50)])
def test_forget_decode_of_many_sequences(cuda_device, dtype, H, D, E, B):
    """More heads than CTAs, fresh and continued sequences and padding rows: the one-token kernels equal the scan."""
    geo, dev = RecurrentGeometry(H, D, E, silu=True, gated=False, form="forget"), cuda_device
    q, v, z = forget_case(H, D, E, B, 3)
    proj = torch.cat([padded(q, geo.kp), padded(v, geo.vp)], 1).to(dtype).to(dev)
    mix = ForgetMix(padded(z, geo.kp).to(dev), columns(rand(H, D, seed=8), geo.kp, dev), columns(rand(H, D, seed=4).sigmoid(), geo.kp, dev))
    norm = columns(rand(H, E, seed=9) + 1.0, geo.vp, dev)
    states = [RecurrentState.zeros(geo, B + 3, dev) for _ in range(2)]
    start = torch.zeros(B + 3, H, geo.kp, geo.vp)
    start[:, :, :D, :E] = rand(B + 3, H, D, E, seed=5)
    for s in states:
        s.s.copy_(start.view(B + 3, H, geo.kp, geo.tiles, 32).permute(0, 1, 3, 2, 4))
    slots = (torch.randperm(B, generator=torch.Generator().manual_seed(1)) + 2).int()
    lens = torch.where(torch.arange(B) % 5 == 3, 1, 20).int()
    if B > 2:
        slots[B // 2], slots[B - 1] = -1, -1
    slots, lens = slots.to(dev), lens.to(dev)
    o, outs = torch.zeros(B, H * geo.vp, device=dev), [torch.zeros(B, H * geo.vp, dtype=dtype, device=dev) for _ in range(2)]
    ops.recurrent_scan(proj, None, geo, None, None, None, 1.0, states[0], slots, torch.arange(B + 1, dtype=torch.int32, device=dev), lens, o, B, B, mix=mix)
    ops.gated_norm(o, norm, None, geo, 1e-5, outs[0], True)
    ops.time_mix_decode(proj, geo, mix, states[1], slots, lens, norm, 1e-5, outs[1], B)
    ops.check_status()
    close(outs[1], outs[0].cpu(), dtype)
    close(states[1].s, states[0].s.cpu(), torch.float32)
    assert B <= 2 or outs[1][B - 1].abs().max() == 0


# ------------------------------------------------------------------------------------------ delta rule
#            heads, kv, dim, vdim, taps
DELTA = [(4, 2, 24, 20, 4), (1, 1, 7, 70, 2), (6, 2, 64, 64, 1), (4, 4, 128, 128, 3), (2, 1, 100, 200, 5), (3, 3, 64, 33, 9), (2, 2, 150, 40, 4)]


def delta_case(shape, n, seed):
    """Projections (rounded to bf16) and logits [step size | decay]: decays between nothing and nearly everything, step sizes up to one, keys that
    come back (so that the triangular system is far from the identity) and a value that the last queries look for."""
    H, G, D, E, _ = shape
    q, k, v = (rand(n, c, m, seed=seed + i, dtype=torch.bfloat16) for i, (c, m) in enumerate(((G, D), (G, D), (H, E))))
    small = torch.cat([rand(n, H, seed=seed + 4) * 2 + 1, rand(n, H, seed=seed + 5) * 2 - 5], 1)
    small[::23, H:] += 12                                   # now and then a head forgets all
    if n > 20:
        k[5::7] = k[2]
        k[6::7] = (0.8 * k[3] + 0.2 * k[6::7]).bfloat16()
    if n > 3:
        v[1] *= 5
        q[n - 2:] = k[1] * 2
    return q, k.bfloat16(), v.bfloat16(), small


def delta_oracle(shape, case, taps, rate, dt_bias):
    H, G, D, E, _ = shape
    q, k, v = (oracle.silu(oracle.causal_conv(x.double().flatten(1), t.double())).view(len(x), -1, c) for x, t, c in zip(case, taps, (D, D, E)))
    q, k = oracle.unit(q).repeat_interleave(H // G, 1) * D ** -0.5, oracle.unit(k).repeat_interleave(H // G, 1)
    small = case[3].double()
    g = torch.exp(-rate.double() * oracle.softplus(small[:, H:] + dt_bias.double()))
    return oracle.delta_scan(q, k, v, g, torch.sigmoid(small[:, :H]))


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", DELTA)
def test_delta_rule_in_portions_slots_and_batches(place, shape):
    """Convolutions behind dirty histories, shared queries and keys, the recurrence in portions that straddle chunk borders, down to two tokens,
    then single tokens, in dirty slots: scan, decode kernel and chunks."""
    dev, dt = place
    H, G, D, E, n_taps = shape
    geo = RecurrentGeometry(H, D, E, silu=False, gated=False, form="delta", groups=G)
    taps = [rand(c, n_taps, seed=40 + i) for i, c in enumerate((G * D, G * D, H * E))]
    rate, dt_bias = rand(H, seed=60).exp(), rand(H, seed=61)
    data = [delta_case(shape, m, 10 * b + 100) for b, m in enumerate(LENS)]
    want = [delta_oracle(shape, d, taps, rate, dt_bias) for d in data]
    conv = torch.cat([padded(t.T.reshape(n_taps, c, -1), p) for t, c, p in zip(taps, (G, G, H), (geo.kp, geo.kp, geo.vp))], 1).contiguous().to(dev)
    state = RecurrentState.zeros(geo, 6, dev)
    state.s.fill_(7.0)
    history = torch.full((6, n_taps - 1, geo.channels), 9.0, dtype=dt, device=dev) if n_taps > 1 else None
    got, bt = [[] for _ in LENS], Batches(LENS, SLOTS, dev)
    for parts in STEPS:
        b = bt.step(parts, dt == torch.bfloat16 and dev == "cuda" and delta_chunked_supported(geo))
        q, k, v, small = (b.rows([d[i] for d in data]) for i in range(4))
        proj = torch.cat([padded(q, geo.kp), padded(k, geo.kp), padded(v, geo.vp), torch.full((b.T, H * geo.vp), 5.0)], 1).to(dt).to(dev)
        small = torch.cat([small, torch.full((b.T, 3), 9.0)], 1).to(dev)
        rows = torch.full((b.T, geo.channels), 3.0, dtype=dt, device=dev)
        rule = DeltaRule(torch.empty(b.T, 2 * G, device=dev), torch.empty(b.T, 2 * H, device=dev))
        alone = b.single == len(b.order)
        ops.delta_rows(proj, small, geo, conv, history, None if alone else b.cut, b.positions, b.state_slots, rate.to(dev), dt_bias.to(dev), rows, rule)
        out = torch.full((b.T, H * geo.vp), 9.0, device=dev)
        a = (rows, None, geo, None, None, None, 1.0, state, b.state_slots)
        if b.single:
            ops.recurrent_scan(*a, None, b.seq_lens, out, b.single, b.single, mix=rule)
        if b.short > b.single:
            ops.recurrent_scan(*a, b.cut, b.seq_lens, out, b.cu[b.short], b.short, b.single, mix=rule)
        if b.table is not None:
            room = torch.empty(delta_workspace(b.table.chunks.shape[0], geo), dtype=torch.uint8, device=dev)
            ops.delta_chunks(rows, geo, rule, state, b.state_slots, b.cut, b.seq_lens, out, b.table, room)
        b.split(out, got)
    for i, m in enumerate(LENS):
        o = torch.cat(got[i]).view(m, H, geo.vp)
        assert geo.vp == E or o[..., E:].abs().max() == 0
        close(o[..., :E], want[i], dt, (shape, i), 3e-2 if dt == torch.bfloat16 else None)
    for part in (1, 3):         # slots nobody owns keep what they held
        assert (state.s[part] == 7.0).all() and (history is None or (history[part] == 9.0).all())


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,E", [(6, 6, 64, 64), (4, 2, 128, 192), (3, 1, 40, 128), (2, 2, 128, 64)])
def test_delta_chunks_equal_the_scan(cuda_device, H, G, D, E):
    """Sequences of one chunk and of many, fresh and continued: outputs and states equal the token-by-token form's on the same rows."""
    geo, dev = RecurrentGeometry(H, D, E, silu=False, gated=False, form="delta", groups=G), cuda_device
    lens, done = [17, 128, 129, 900, 40, 2000], [0, 5, 0, 300, 64, 0]
    cu = [0]
    for m in lens:
        cu.append(cu[-1] + m)
    T = cu[-1]
    q, k, v, small = delta_case((H, G, D, E, 1), T, 3)
    rows = torch.cat([padded(q, geo.kp), padded(k, geo.kp), padded(v, geo.vp)], 1).to(dev)
    rule = DeltaRule(torch.cat([1 / q.float().norm(dim=-1), 1 / k.float().norm(dim=-1)], 1).to(dev),
                     torch.cat([-torch.nn.functional.softplus(small[:, H:]), torch.sigmoid(small[:, :H])], 1).to(dev))
    states = [RecurrentState.zeros(geo, 8, dev) for _ in range(2)]
    start = torch.zeros(8, H, geo.kp, geo.vp)
    start[:, :, :D, :E] = rand(8, H, D, E, seed=5)
    for s in states:
        s.s.copy_(start.view(8, H, geo.kp, geo.tiles, 32).permute(0, 1, 3, 2, 4))
    slots, lens_t, cut = i32([7, 3, 0, 5, 1, 2], dev), i32([a + b for a, b in zip(lens, done)], dev), i32(cu, dev)
    outs = [torch.zeros(T, H * geo.vp, device=dev) for _ in range(2)]
    ops.recurrent_scan(rows, None, geo, None, None, None, 1.0, states[0], slots, cut, lens_t, outs[0], T, 6, mix=rule)
    table = ChunkTable.make(cu, 0, dev)
    room = torch.empty(delta_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device=dev)
    for _ in range(2):          # (twice: nothing is left behind in the workspace)
        states[1].s.copy_(start.view(8, H, geo.kp, geo.tiles, 32).permute(0, 1, 3, 2, 4))
        ops.delta_chunks(rows, geo, rule, states[1], slots, cut, lens_t, outs[1], table, room)
        ops.check_status()
        close(outs[1], outs[0].cpu(), torch.bfloat16)
        close(states[1].s, states[0].s.cpu(), torch.float32, tol=1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,B", [(6, 3, 40, 64, 300), (16, 16, 128, 128, 64), (1, 1, 64, 30, 1), (4, 2, 300, 70, 50)])
def test_delta_decode_of_many_sequences(cuda_device, dtype, H, G, D, E, B):
    """More tiles than CTAs, fresh and continued sequences and padding rows: the one-token kernels equal the scan."""
    geo, dev = RecurrentGeometry(H, D, E, silu=False, gated=False, form="delta", groups=G), cuda_device
    q, k, v, small = delta_case((H, G, D, E, 1), B, 3)
    rows = torch.cat([padded(q, geo.kp), padded(k, geo.kp), padded(v, geo.vp)], 1).to(dtype).to(dev)
    rule = DeltaRule(torch.cat([1 / q.float().norm(dim=-1), 1 / k.float().norm(dim=-1)], 1).to(dev),
                     torch.cat([-torch.nn.functional.softplus(small[:, H:]), torch.sigmoid(small[:, :H])], 1).to(dev))
    states = [RecurrentState.zeros(geo, B + 3, dev) for _ in range(2)]
    for s in states:
        s.s[:, :, :, :D] = rand(*s.s.shape, seed=5)[:, :, :, :D].to(dev)
    slots = (torch.randperm(B, generator=torch.Generator().manual_seed(1)) + 2).int()
    lens = torch.where(torch.arange(B) % 5 == 3, 1, 20).int()
    if B > 2:
        slots[B // 2], slots[B - 1] = -1, -1
    slots, lens = slots.to(dev), lens.to(dev)
    outs = [torch.zeros(B, H * geo.vp, device=dev) for _ in range(2)]
    a = (rows, None, geo, None, None, None, 1.0)
    ops.recurrent_scan(*a, states[0], slots, torch.arange(B + 1, dtype=torch.int32, device=dev), lens, outs[0], B, B, mix=rule)
    ops.recurrent_scan(*a, states[1], slots, None, lens, outs[1], B, B, mix=rule)
    ops.check_status()
    close(outs[1], outs[0].cpu(), torch.float32)
    close(states[1].s, states[0].s.cpu(), torch.float32)
    assert B <= 2 or outs[1][B - 1].abs().max() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", DELTA)
def test_delta_rows_of_a_large_batch(cuda_device, dtype, shape):
    """Hundreds of rows of unlike sequences at once, some behind a history, one without a slot: as the CPU twin."""
    H, G, D, E, n_taps = shape
    geo = RecurrentGeometry(H, D, E, silu=False, gated=False, form="delta", groups=G)
    lens, done = [1, 2, 1, 3, 700, 290, 7, 1005], [0, 4, 1, 0, 0, 33, 2, 0]
    cu = [0]
    for m in lens:
        cu.append(cu[-1] + m)
    T = cu[-1]
    proj, small = rand(T, geo.proj, seed=1, dtype=torch.bfloat16), rand(T, 2 * H + 1, seed=2)
    conv, rate, dt_bias = rand(n_taps, geo.channels, seed=3), rand(H, seed=4).exp(), rand(H, seed=5)
    positions = torch.cat([torch.arange(d, d + m) for m, d in zip(lens, done)]).int()
    slots, res = i32([6, 2, 0, 8, 1, 3, 9, -1]), []
    for dev, dt in (("cpu", torch.float32), (cuda_device, dtype)):
        history = rand(10, n_taps - 1, geo.channels, seed=6, dtype=torch.bfloat16).to(dt).to(dev) if n_taps > 1 else None
        rows, rule = torch.zeros(T, geo.channels, dtype=dt, device=dev), DeltaRule(torch.zeros(T, 2 * G, device=dev), torch.zeros(T, 2 * H, device=dev))
        ops.delta_rows(proj.to(dt).to(dev), small.to(dev), geo, conv.to(dev), history, i32(cu, dev), positions.to(dev), slots.to(dev), rate.to(dev),
                       dt_bias.to(dev), rows, rule)
        res.append((rows, rule.units, rule.steps, history))
    end = T - 1005              # (the twin leaves a sequence without a slot alone)
    for what, want, got in zip(("rows", "units", "steps"), *res):
        close(got[:end], want[:end], dtype, what)
    if n_taps > 1:
        close(res[1][3], res[0][3], dtype)


# ------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", [(6, 2, 24, 40, 12), (3, 3, 20, 13, 20), (8, 1, 128, 64, 64), (2, 1, 64, 128, 16), (2, 2, 130, 72, 2)])
def test_temperature_of_a_head(place, shape):
    """Queries times their head's number after the rotation; keys as they are."""
    dev, dt = place
    H, G, D, E, rot = shape
    geo = GroupedGeometry(H, G, D, E, rot_dims=rot, window=9, temperature=True)
    spec, T = {"dims": rot, "base": 400.0}, 40
    q, k, v = (rand(T, n, c, seed=1 + i, dtype=torch.bfloat16) for i, (n, c) in enumerate(((H, D), (G, D), (G, E))))
    temp = rand(H, seed=9) + 1.5
    proj = torch.zeros(T, geo.proj)
    proj[:, :H * D], proj[:, geo.k_col:geo.k_col + G * D], proj[:, geo.v_col:geo.v_col + G * E] = q.flatten(1), k.flatten(1), v.flatten(1)
    cache = GroupedCache(*(torch.zeros(3, G, KV_BLOCK, geo.dp, dtype=dt, device=dev) for _ in range(2)), None)
    at = torch.arange(T)
    got = torch.zeros(T, H * geo.dp, dtype=dt, device=dev)
    table = ops.frequency_table(T, [400.0 ** (-2 * i / rot) for i in range(rot // 2)], 1.0, dev)
    ops.grouped_append(proj.to(dt).to(dev), geo, conv=None, cache=cache, cu_q=i32([0, T], dev), positions=at.int().to(dev), state_slots=i32([0], dev),
                       slots=at.int().to(dev), q_norm=None, k_norm=None, eps=1e-5, table=table, q=got, q_factor=temp.to(dev))
    close(got.view(T, H, geo.dp)[..., :D], oracle.rotate(q.double(), spec) * temp.double()[:, None], dt)
    close(cache.keys[at // KV_BLOCK, :, at % KV_BLOCK, :D], oracle.rotate(k.double(), spec), dt)
    out = torch.zeros(T, H * geo.dp, dtype=dt, device=dev)
    ops.grouped_attention(got, geo, cache, i32([[0, 1, 2]], dev), i32([0, T], dev), i32([T], dev), out, scale=0.3, rows=T, max_q=T, n_single=0)
    want = oracle.attend(oracle.rotate(q.double(), spec), oracle.rotate(k.double(), spec), v.double(), 0.3 * temp.double(), oracle.seen_window(T, 9))
    close(out.view(T, H, geo.dp)[..., :E], want, dt, tol=2e-2 if dt == torch.bfloat16 else None)


# ------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T,n", [(5, 40), (3, 13), (130, 1024), (2, 6144)])
def test_normed_powers(place, T, n):
    dev, dt = place
    p = -(-n // 8) * 8
    z = torch.zeros(T, p)
    z[:, :n] = rand(T, n, seed=1, dtype=torch.bfloat16) * torch.linspace(0.01, 4, T)[:, None].bfloat16()
    act = torch.tensor([0.4, -0.7, 0.9, 0.3])
    out = torch.full((T, p), 9.0, dtype=dt, device=dev)
    ops.poly_norm(z.to(dt).to(dev), act.to(dev), n, 1e-3, out)
    close(out[:, :n], oracle.poly_norm(z[:, :n].to(dt).double(), act.double(), 1e-3), dt)
    assert p == n or out[:, n:].abs().max() == 0


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("experts,identity,top,ff,d,T", [(5, 2, 3, 40, 56, 33), (1, 1, 1, 8, 24, 3), (12, 0, 12, 17, 30, 5), (60, 9, 8, 192, 128, 300), (3, 5, 8, 30, 64, 150)])
def test_experts_with_corrected_choices_and_identities(place, experts, identity, top, ff, d, T):
    """The correction picks, the plain softmax score weighs, some choices hand the input on; through the stream with a gated shared output.
    Twice with one scratch: the histogram is left empty."""
    dev, dt = place
    width, n = -(-d // 8) * 8, experts + identity
    geo = ExpertsGeometry.make(experts, top, ff, width, None, dt, normalize=False, identity=identity)
    w = {}
    for e in range(experts):
        for part, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
            w[f"m.e{e}.{part}"] = (rand(*shape, seed=7 * e + len(part)) * 2 / shape[1] ** 0.5).bfloat16()
    wgu = torch.zeros(experts * 2 * geo.ffp, width, dtype=dt, device=dev)
    wd = torch.zeros(experts * width, geo.ffp, dtype=dt, device=dev)
    ops.pack_experts(*([w[f"m.e{e}.{part}"].to(dev) for e in range(experts)] for part in ("gate", "up", "down")), geo, wgu, wd)
    scratch = ExpertsScratch(geo, T + 5, dt, torch.device(dev))
    scratch.y.fill_(float("nan"))                        # (rows of choices that are no experts are never read)
    correction = rand(n, seed=77).abs() * 0.5
    post = ops.StreamNorm(torch.ones(width, device=dev))
    for seed in (1, 2):
        h, z, shared = rand(T, d, seed=seed, dtype=torch.bfloat16), rand(T, n + 1, seed=seed + 10) * 2, rand(T, d, seed=seed + 20)
        hp, sp = torch.zeros(T, width, dtype=dt), torch.zeros(T, width)
        hp[:, :d], sp[:, :d] = h, shared
        hp, small = hp.to(dev), torch.cat([z, torch.full((T, 2), 99.0)], 1).to(dev)
        y, p = ops.experts_forward(hp, small, geo, scratch, wgu, wd, correction.to(dev))
        x = torch.zeros(T, width, device=dev)
        ops.stream_sandwich(x, d, y=sp.to(dev), gate=small[:, n:], chosen=ops.ChosenExperts(y, p, scratch.idx[:T], experts, hp), post=post, eps=1e-5)
        wz, want = {k: v.double() for k, v in w.items()}, torch.sigmoid(z[:, n:].double()) * shared.double()
        best, pw = oracle.route(z[:, :n].double(), correction.double(), top)
        for e in range(n):
            t, j = (best == e).nonzero(as_tuple=True)
            want[t] += pw[t, j, None] * (oracle.gated_unit(h[t].double(), wz, f"m.e{e}") if e < experts else h[t].double())
        close(x[:, :d], oracle.rms(want, 1e-5), dt)
        assert width == d or x[:, d:].abs().max() == 0
    idx, pw = route_reference(torch.tensor([[1.0, 0.9, 0.0]]), 1, normalize=False, correction=torch.tensor([0.0, 0.5, 0.0]))
    assert idx.item() == 1 and abs(pw.item() - torch.tensor([1.0, 0.9, 0.0]).softmax(0)[1].item()) < 1e-6


# ------------------------------------------------------------------------------------------ stream
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("bounded", [True, False])
@pytest.mark.parametrize("d", [30, 200, 2048])
def test_stream_between_norms(place, bounded, d):
    """One sublayer's output, or two normed halves; both kinds of norm; and the last rows alone."""
    dev, dt = place
    p, eps = -(-d // 8) * 8, 1e-3

    def pad(x):
        out = torch.zeros(*x.shape[:-1], p)
        out[..., :d] = x
        return out.to(dev)

    w = {}
    for i, name in enumerate(("post", "pre")):
        w[name] = rand(d, seed=5 + i) + 1
        if bounded:
            w[name + ".b"], w[name + ".alpha"] = rand(d, seed=7 + i), torch.tensor(0.4 + i)
    wd = {k: v.double() for k, v in w.items()}

    def norm(x, name):
        return oracle.bounded(x, wd, name) if bounded else oracle.rms(x, eps) * wd[name]

    norms = {n: ops.StreamNorm(pad(w[n]), pad(w[n + ".b"]) if bounded else None, w[n + ".alpha"].view(1).to(dev) if bounded else None) for n in ("post", "pre")}
    x, y, y2, wl, wr = rand(6, d, seed=1), rand(6, d, seed=2) * 3, rand(6, d, seed=3) * 0.05, rand(d, seed=8), rand(d, seed=9)
    for pair in (False, True):
        v = y.double() if not pair else (oracle.rms(y.double(), eps) * wl.double() + oracle.rms(y2.double(), eps) * wr.double()) / 2
        want = x.double() + norm(v, "post")
        xs, h, copy = pad(x), torch.zeros(6, p, dtype=dt, device=dev), torch.zeros(6, 2 * p, dtype=dt, device=dev)
        ops.stream_sandwich(xs, d, y=pad(y), pair=(pad(y2), pad(wl), pad(wr)) if pair else None, post=norms["post"], pre=norms["pre"], eps=eps,
                            copy=copy[:, :p], h=h)
        close(xs[:, :d], want, torch.float32)
        close(copy[:, :d], want, dt)
        close(h[:, :d], norm(want, "pre"), dt)
        assert p == d or (xs[:, d:].abs().max() == 0 and h[:, d:].abs().max() == 0)
    rows = torch.tensor([5, 0, 0], dtype=torch.int32)
    out = torch.zeros(3, p, dtype=dt, device=dev)
    ops.stream_sandwich(xs, d, pre=norms["pre"], eps=eps, h=out, rows=rows.to(dev))
    close(out[:, :d], norm(want, "pre")[rows.long()], dt)
    close(xs[:, :d], want, torch.float32)

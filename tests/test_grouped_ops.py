"""The operations behind the Fogurax design one by one against the plain oracle (``fogurax_oracle.py``): CPU twins, and on a GPU the
kernels in bf16 and fp32. Attention carries planted keys just inside and just outside of what a query sees, time mixing a token
that late queries look for, convolutions dirty histories, so that an edge that is off by one or a lost state shows."""

import math

import fogurax_oracle as oracle
import pytest
import torch
from test_recurrent_ops import PLACES, close, i32, padded, rand

from research_b200 import ops
from research_b200.models.stack import BandScaling, RotarySpec, YarnScaling
from research_b200.ops.experts import ExpertsGeometry, ExpertsScratch
from research_b200.ops.grouped import KV_BLOCK, GroupedCache, GroupedGeometry
from research_b200.ops.recurrent import ChunkTable, RecurrentGeometry, RecurrentState, TimeMix, time_mix_chunked_supported, time_mix_workspace


# ------------------------------------------------------------------------------------------ rotations
@pytest.mark.parametrize("dims,base,original", [(16, 1e4, 64), (40, 5e5, 300), (2, 100.0, 50), (64, 1e4, 2048)])
def test_frequencies(dims, base, original):
    plain = {"dims": dims, "base": base}
    band = {"factor": 5.0, "low": 1.5, "high": 6.0, "original": original}
    yarn = {"factor": 3.0, "original": original, "fast": 20.0, "slow": 0.5}
    for scaling, rule in ((BandScaling(**band), oracle.band_frequencies), (YarnScaling(**yarn), oracle.yarn_frequencies), (None, oracle.plain_frequencies)):
        rot = RotarySpec(dims, base, True, scaling)
        want = rule({**plain, "scaling": band if rule is oracle.band_frequencies else yarn})
        assert torch.allclose(torch.tensor(rot.frequencies(), dtype=torch.float64), torch.tensor(want, dtype=torch.float64), rtol=1e-12)
    if dims >= 40:       # all three bands and a ramp that is neither 0 nor 1 are there
        kept = [a / b for a, b in zip(oracle.band_frequencies({**plain, "scaling": band}), oracle.plain_frequencies(plain))]
        assert kept[0] == 1 and abs(kept[-1] - 0.2) < 1e-9 and any(0.21 < k < 0.99 for k in kept)
        ramp = [a / b for a, b in zip(oracle.yarn_frequencies({**plain, "scaling": yarn}), oracle.plain_frequencies(plain))]
        assert any(0.35 < r < 0.98 for r in ramp)
    table = ops.frequency_table(5, [0.5, 2.0], 1.25)
    assert torch.allclose(table[3], 1.25 * torch.tensor([[math.cos(1.5), math.sin(1.5)], [math.cos(6.0), math.sin(6.0)]]))


# ------------------------------------------------------------------------------------------ projection to queries, keys and values
#        heads, kv, dim, vdim, taps, conv, norm, rotated, interleaved
APPENDS = [(6, 2, 24, 40, 3, True, "head", 16, True), (3, 3, 20, 13, 1, False, "projection", 20, False), (1, 1, 7, 5, 4, True, "", 2, True),
           (8, 1, 128, 128, 2, True, "head", 64, True), (4, 2, 64, 24, 1, True, "projection", 0, True), (2, 1, 300, 72, 5, True, "head", 100, False),
           (40, 8, 32, 32, 1, False, "projection", 32, False)]


def conved(u, taps):
    return oracle.causal_conv(u, taps) if taps is not None else u


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", APPENDS)
def test_append_in_portions(place, shape):
    """Four sequences in portions down to one token, in slots whose histories hold something else: every query, cached key and value
    equals the whole sequence's."""
    dev, dt = place
    H, G, D, E, taps, conv, norm, rot, inter = shape
    geo = GroupedGeometry(H, G, D, E, taps, conv, norm, rot, inter)
    lens, eps, nb = [37, 5, 64, 18], 1e-4, 16
    spec = RotarySpec(max(rot, 2), 300.0, inter, BandScaling(4.0, 1.0, 3.0, 30))
    freq = spec.frequencies() if rot else []
    table = ops.frequency_table(80, freq, 1.3, dev) if rot else torch.zeros(80, 0, 2, device=dev)
    taps_w = {n: rand(c, taps, seed=5 + i) if conv else None for i, (n, c) in enumerate((("q", H * D), ("k", G * D), ("v", G * E)))}
    qn, kn = (rand(n * D, seed=8 + i) + 1.5 if norm == "projection" else None for i, n in enumerate((H, G)))
    data, want = [], []
    for b, n in enumerate(lens):
        u = {x: rand(n, c, seed=20 + 5 * b + i, dtype=torch.bfloat16) for i, (x, c) in enumerate((("q", H * D), ("k", G * D), ("v", G * E)))}
        row = torch.zeros(n, geo.proj)
        row[:, :H * D], row[:, geo.k_col:geo.k_col + G * D], row[:, geo.v_col:geo.v_col + G * E] = u["q"], u["k"], u["v"]
        data.append(row.to(dt))
        out = []
        for x, heads, w in (("q", H, qn), ("k", G, kn)):
            y = conved(u[x].double(), taps_w[x].double() if conv else None)
            if norm == "projection":
                y = oracle.rms(y, eps) * w.double()
            y = oracle.rotate(y.view(n, heads, D), freq, 1.3, inter)
            out.append(oracle.rms(y, eps) if norm == "head" else y)
        want.append((*out, conved(u["v"].double(), taps_w["v"].double() if conv else None).view(n, G, E)))
    weights = None
    if conv:
        weights = torch.zeros(taps, geo.channels, device=dev)
        for x, col in (("q", 0), ("k", geo.k_col), ("v", geo.v_col)):
            weights[:, col:col + taps_w[x].shape[0]] = taps_w[x].T.to(dev)
    cache = GroupedCache(*(torch.zeros(nb, G, KV_BLOCK, geo.dp, dtype=dt, device=dev) for _ in range(2)),
                         torch.full((7, taps - 1, geo.channels), 9.0, dtype=dt, device=dev) if taps > 1 else None)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(2))
    blocks = [perm[4 * b:4 * b + 4] for b in range(4)]
    slots, done, got = [5, 0, 6, 2], [0] * 4, [[] for _ in lens]

    def step(parts, decode=False):
        rows = torch.cat([data[b][done[b]:done[b] + n] for b, n in parts.items()]).to(dev)
        pos = torch.cat([torch.arange(done[b], done[b] + n) for b, n in parts.items()])
        place_of = torch.cat([blocks[b][torch.arange(done[b], done[b] + n) // KV_BLOCK] for b, n in parts.items()]) * KV_BLOCK + pos % KV_BLOCK
        cu = [0]
        for n in parts.values():
            cu.append(cu[-1] + n)
        q = torch.full((cu[-1], H * geo.dp), 7.0, dtype=dt, device=dev)
        ops.grouped_append(rows, geo, conv=weights, cache=cache, cu_q=None if decode else i32(cu, dev), positions=pos.int().to(dev),
                           state_slots=i32([slots[b] for b in parts], dev), slots=place_of.int().to(dev), q_norm=qn.to(dev) if qn is not None else None,
                           k_norm=kn.to(dev) if kn is not None else None, eps=eps, table=table, q=q)
        for i, (b, n) in enumerate(parts.items()):
            got[b].append(q[cu[i]:cu[i + 1]].cpu())
            done[b] += n

    step({0: 2, 2: 30})
    step({1: 1, 0: 7, 3: 2})
    step({0: 1, 1: 1, 2: 1, 3: 1}, decode=True)
    step({3: 1, 1: 3, 0: 11, 2: 2})
    step({0: 1, 3: 1}, decode=True)
    step({0: 15, 2: 31, 3: 13})
    assert done == lens
    for b, n in enumerate(lens):
        q = torch.cat(got[b]).view(n, H, geo.dp)
        at = torch.arange(n)
        k, v = (c[blocks[b][at // KV_BLOCK], :, at % KV_BLOCK].cpu() for c in (cache.keys, cache.values))
        for x, y, size in ((q, want[b][0], D), (k, want[b][1], D), (v, want[b][2], E)):
            close(x[..., :size], y, dt, (shape, b))
            assert size == geo.dp or x[..., size:].abs().max() == 0
    if taps > 1:
        free = [s for s in range(7) if s not in slots]
        assert (cache.history[free] == 9.0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", APPENDS)
def test_append_of_a_large_batch(cuda_device, dtype, shape):
    """Hundreds of rows of unlike sequences at once, some behind a history, some without a place in the cache: as the CPU twin."""
    H, G, D, E, taps, conv, norm, rot, inter = shape
    geo = GroupedGeometry(H, G, D, E, taps, conv, norm, rot, inter)
    lens, done, nb = [1, 2, 1, 3, 300, 290, 7, 5], [0, 4, 1, 0, 0, 33, 2, 0], 60
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    T = cu[-1]
    proj = torch.zeros(T, geo.proj)
    for col, n in ((0, H * D), (geo.k_col, G * D), (geo.v_col, G * E)):
        proj[:, col:col + n] = rand(T, n, seed=col + 1, dtype=torch.bfloat16)
    slots = torch.randperm(nb * KV_BLOCK, generator=torch.Generator().manual_seed(3))[:T].int()
    slots[::9] = -1
    positions = torch.cat([torch.arange(d, d + n) for n, d in zip(lens, done)]).int()
    state_slots = torch.tensor([6, 2, 0, 8, 1, 3, 9, 5], dtype=torch.int32)
    weights = rand(taps, geo.channels, seed=7) if conv else None
    qn, kn = (rand(n * D, seed=8 + i) + 1.5 if norm == "projection" else None for i, n in enumerate((H, G)))
    table = ops.frequency_table(400, [0.9 ** i for i in range(rot // 2)], 1.2)
    res = []
    for dev, dt in (("cpu", torch.float32), (cuda_device, dtype)):
        cache = GroupedCache(*(torch.zeros(nb, G, KV_BLOCK, geo.dp, dtype=dt, device=dev) for _ in range(2)),
                             rand(10, taps - 1, geo.channels, seed=4, dtype=torch.bfloat16).to(dt).to(dev) if taps > 1 else None)
        q = torch.zeros(T, H * geo.dp, dtype=dt, device=dev)
        to = lambda t: t.to(dev) if t is not None else None
        ops.grouped_append(proj.to(dt).to(dev), geo, conv=to(weights), cache=cache, cu_q=i32(cu, dev), positions=to(positions), state_slots=to(state_slots),
                           slots=to(slots), q_norm=to(qn), k_norm=to(kn), eps=1e-4, table=to(table), q=q)
        res.append((q, cache.keys, cache.values) + ((cache.history,) if taps > 1 else ()))
    for want, got in zip(*res):
        close(got, want, dtype)


@pytest.mark.parametrize("place", PLACES)
def test_append_skips_padding_rows(place):
    dev, dt = place
    geo = GroupedGeometry(2, 1, 8, 8, 3, True, "head", 4, True)
    cache = GroupedCache(*(torch.full((2, 1, KV_BLOCK, 64), 3.0, dtype=dt, device=dev) for _ in range(2)),
                         torch.full((4, 2, geo.channels), 9.0, dtype=dt, device=dev))
    q = torch.zeros(3, 128, dtype=dt, device=dev)
    ops.grouped_append(torch.ones(3, geo.proj, dtype=dt, device=dev), geo, conv=torch.ones(3, geo.channels, device=dev), cache=cache, cu_q=None,
                       positions=i32([0, 0, 4], dev), state_slots=i32([-1, 1, -1], dev), slots=i32([-1, 17, -1], dev), q_norm=None, k_norm=None, eps=1e-6,
                       table=ops.frequency_table(8, [1.0, 0.5], 1.0, dev), q=q)
    assert int((cache.keys == 3.0).all(-1).sum()) == 31 and int((cache.values == 3.0).any(-1).sum()) == 32
    assert (cache.history[[0, 2, 3]] == 9.0).all() and (cache.history[1, 0] == 1.0).all()


# ------------------------------------------------------------------------------------------ attention
SEEN = {"all": {}, "window": {"window": 45}, "chunk": {"chunk": 50}, "window1": {"window": 1}, "block": {"chunk": 16}, "wide": {"window": 200}}


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", [(6, 2, 24, 40), (1, 1, 7, 64), (8, 1, 128, 128), (40, 2, 64, 20), (4, 4, 136, 200)])
@pytest.mark.parametrize("span", list(SEEN))
def test_attention_sees_what_it_should(place, shape, span):
    """Scattered blocks, prompts, portions behind cached tokens and single tokens in one batch. For a number of queries the key just inside
    and the key just outside of their reach stand out with a value of their own."""
    dev, dt = place
    H, G, D, E = shape
    geo = GroupedGeometry(H, G, D, E, rot_dims=2, **SEEN[span])
    scale, factor, splits = 1.2 * D ** -0.5, 0.7, 3
    lens, done, nb = [70, 300, 33, 51, 130, 257], [69, 299, 32, 50, 0, 100], 80
    perm, at = torch.randperm(nb, generator=torch.Generator().manual_seed(1)), 0
    cache = GroupedCache(*(torch.zeros(nb, G, KV_BLOCK, geo.dp, dtype=dt, device=dev) for _ in range(2)), None)
    tables, new_q, gates, wants = torch.zeros(6, 24, dtype=torch.int32), [], [], []
    for b, (L, d0) in enumerate(zip(lens, done)):
        q, k, v = (rand(L, n, c, seed=30 + 3 * b + i, dtype=torch.bfloat16) for i, (n, c) in enumerate(((H, D), (G, D), (G, E))))
        seen = {"window": oracle.seen_window, "chunk": oracle.seen_chunk}
        mask = next((seen[kind](L, size) for kind, size in SEEN[span].items()), oracle.seen_causal(L))
        for i, p in enumerate({L - 1, L - 2, d0 + (L - d0) // 2, min(d0 + 17, L - 1)}):
            first = int(mask[p].nonzero()[0])
            for j in (first, first - 1, p):
                if j >= 0:
                    k[j] = rand(G, D, seed=90 + 10 * b + i).sign().bfloat16()
                    v[j] += 3 * (1 + j - first)
            q[p] = 2 * k[first].repeat_interleave(H // G, 0)
        gate = rand(L, H, seed=60 + b)
        o = oracle.attend(q.double(), k.double(), v.double(), scale, mask) * torch.sigmoid(gate.double())[..., None] * factor
        wants.append(o[d0:])
        nblk = -(-L // KV_BLOCK)
        tables[b, :nblk] = perm[at:at + nblk]
        at += nblk
        pos = torch.arange(L)
        blk = tables[b, pos // KV_BLOCK].long()
        for c, x, n in ((cache.keys, k, D), (cache.values, v, E)):
            c[blk, :, pos % KV_BLOCK, :n] = x.to(dt).to(dev)
        new_q.append(padded(q[d0:].float(), geo.dp))
        gates.append(gate[d0:])
    cu = [0]
    for L, d0 in zip(lens, done):
        cu.append(cu[-1] + L - d0)
    q, T = torch.cat(new_q).to(dt).to(dev), cu[-1]
    gate = torch.cat([torch.cat(gates), torch.full((T, 3), 50.0)], 1).to(dev)
    out = torch.full((T, H * geo.dp + 16), 5.0, dtype=dt, device=dev)
    ws = torch.zeros(ops.kv_workspace(geo, 6, splits), device=dev)
    args = dict(scale=scale, gate_scale=factor, workspace=ws, splits=splits)
    ops.grouped_attention(q, geo, cache, tables.to(dev), i32(cu, dev), i32(lens, dev), out[:, :H * geo.dp], rows=T, max_q=157, n_single=4, gate=gate, **args)
    assert (out[:, H * geo.dp:] == 5.0).all()
    for b in range(6):
        got = out[cu[b]:cu[b + 1], :H * geo.dp].reshape(-1, H, geo.dp)
        close(got[..., :E], wants[b], dt, (shape, span, b), 2e-2 if dt == torch.bfloat16 else None)
        assert E == geo.dp or got[..., E:].abs().max() == 0
    dec = torch.full((5, H * geo.dp), 5.0, dtype=dt, device=dev)      # the same single tokens as a decode batch with a padding row
    ops.grouped_attention(torch.cat([q[:4], q[:1]]), geo, cache, torch.cat([tables[:4], tables[:1]]).to(dev), None, i32(lens[:4] + [0], dev), dec, rows=5, max_q=1,
                          n_single=5, gate=gate[[0, 1, 2, 3, 0]].contiguous(), **args)
    close(dec[:4], out[:4, :H * geo.dp].cpu(), dt)
    assert dec[4].abs().max() == 0


# ------------------------------------------------------------------------------------------ time mixing
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("width", [8, 40, 2048])
def test_token_shift_in_portions(place, width):
    dev, dt = place
    lens, slots = [9, 1, 30], [3, 0, 1]
    h = [rand(n, width, seed=i, dtype=torch.bfloat16) for i, n in enumerate(lens)]
    mu = rand(5, width, seed=9)
    hist = torch.full((5, 1, width), 9.0, dtype=dt, device=dev)
    got, done = [[] for _ in lens], [0, 0, 0]

    def step(parts, decode=False):
        rows = torch.cat([h[b][done[b]:done[b] + n] for b, n in parts.items()]).to(dt).to(dev)
        pos = torch.cat([torch.arange(done[b], done[b] + n) for b, n in parts.items()]).int().to(dev)
        cu = [0]
        for n in parts.values():
            cu.append(cu[-1] + n)
        out = torch.zeros(5, cu[-1] + 2, width, dtype=dt, device=dev)
        ops.token_shift(rows, mu.to(dev), out, hist, None if decode else i32(cu, dev), pos, i32([slots[b] for b in parts], dev))
        for i, (b, n) in enumerate(parts.items()):
            got[b].append(out[:, cu[i]:cu[i + 1]].cpu())
            done[b] += n

    step({0: 3, 2: 2})
    step({1: 1, 0: 1, 2: 1}, decode=True)
    step({2: 1, 0: 2})
    step({0: 1, 2: 20})
    step({0: 2, 2: 6})
    assert done == lens
    for b in range(3):
        x = h[b].double()
        want = torch.stack([x + (oracle.previous(x) - x) * m.double() for m in mu])
        close(torch.cat(got[b], 1), want, dt)
    assert (hist[[2, 4]] == 9.0).all() and torch.equal(hist[3, 0].cpu(), h[0][-1].to(dt))


@pytest.mark.parametrize("place", PLACES)
def test_tanh_as_exact_operand(place):
    dev, dt = place
    x = rand(30, 24, seed=1)
    out = torch.zeros(30, 24 if dt == torch.float32 else 48, dtype=dt, device=dev)
    ops.tanh_parts(x.to(dev), out)
    got = out.double().cpu()
    got = got if dt == torch.float32 else got[:, :24] + got[:, 24:]
    assert (got - torch.tanh(x.double())).abs().max() < (1e-6 if dt == torch.float32 else 1e-5)


def mix_case(geo, lens, seed, strong):
    """r, k, v, gate and decay logits of several sequences; the second token is found again by the last ones, through channels that keep
    nearly everything. ``strong``: other channels lose all they have within a token."""
    T, H, D = sum(lens), geo.heads, geo.dim
    r, k, v, g = (rand(T, H, D, seed=seed + i, dtype=torch.bfloat16) * (1.0 if i == 2 else 0.5) for i in range(4))
    z = rand(T, H, D, seed=seed + 5) * (2.5 if strong else 0.7) - 1
    slow = torch.arange(D) % 3 == 0
    z[..., slow] = -7 + 0.3 * z[..., slow]
    at = 0
    for n in lens:
        if n > 3:
            mark = torch.where(slow, rand(H, D, seed=seed + 6).sign() * 2, 0).bfloat16()
            k[at + 1] = mark
            r[at + n - 2:at + n] = mark
        at += n
    return r.bfloat16(), k.bfloat16(), v.bfloat16(), g.bfloat16(), z


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("shape", [(3, 24), (1, 7), (5, 64), (2, 128), (2, 90), (1, 200)])
def test_time_mixing_in_portions_slots_and_batches(place, shape, strong):
    """Portions that straddle chunk borders, down to two tokens, then single tokens, in dirty slots: scan, decode kernel and chunks."""
    dev, dt = place
    H, D = shape
    geo = RecurrentGeometry(H, D, D, silu=False, gated=False)
    lens, eps, slots = [150, 60, 273, 9], 1e-4, [4, 0, 5, 2]
    w0, bonus, norm = rand(H, D, seed=50) * 0.5, rand(H, D, seed=51), rand(H * D, seed=52) + 1.5
    data = [mix_case(geo, [n], 10 * b + 100, strong) for b, n in enumerate(lens)]
    want = []
    for r, k, v, g, z in data:
        decay = torch.exp(-torch.exp(z.double() + w0.double()))
        o = oracle.time_mix_scan(r.double(), k.double(), v.double(), decay, bonus.double())
        want.append(oracle.rms(o, eps).flatten(1) * norm.double() * oracle.silu(g.double().flatten(1)))
    state = RecurrentState.zeros(geo, 6, dev)
    state.s.fill_(7.0)
    flat = {k: padded(x.view(1, H, D), geo.kp).view(-1).to(dev) for k, x in (("w0", w0), ("bonus", bonus), ("norm", norm))}
    got = [[] for _ in lens]

    def step(parts):
        order = sorted(parts, key=lambda b: parts[b])
        rows = {b: sum(len(x) for x in got[b]) for b in order}
        cols = [torch.cat([data[b][i][rows[b]:rows[b] + parts[b]] for b in order]) for i in range(5)]
        proj = torch.cat([padded(c, geo.kp) for c in cols[:4]], 1).to(dt).to(dev)
        T, cu = proj.shape[0], [0]
        for b in order:
            cu.append(cu[-1] + parts[b])
        mix = TimeMix(padded(cols[4], geo.kp).to(dev), flat["w0"], flat["bonus"])
        o, out = torch.full((T, H * geo.vp), 9.0, device=dev), torch.full((T, H * geo.vp + 8), 9.0, dtype=dt, device=dev)[:, :H * geo.vp]
        a = (proj, None, geo, None, None, None, 1.0, state, i32([slots[b] for b in order], dev))
        cut, sl = i32(cu, dev), i32([rows[b] + parts[b] for b in order], dev)
        single = next((i for i, b in enumerate(order) if parts[b] > 1), len(order))
        chunks = dt == torch.bfloat16 and dev == "cuda" and time_mix_chunked_supported(geo)
        short = next((i for i, b in enumerate(order) if parts[b] > 16), len(order)) if chunks else len(order)
        if single:
            ops.time_mix_decode(proj, geo, mix, state, a[-1], sl, flat["norm"], eps, out, single)
        if short > single:
            ops.recurrent_scan(*a, cut, sl, o, cu[short], short, single, mix=mix)
            ops.gated_norm(o[single:cu[short]], flat["norm"], proj[single:, geo.offsets[3]:], geo, eps, out[single:], True, silu=True)
        if short < len(order):
            table = ChunkTable.make(cu, short, dev)
            room = torch.empty(time_mix_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device=dev)
            ops.time_mix_chunks(proj, geo, mix, state, a[-1], cut, sl, flat["norm"], eps, out, table, room)
        for i, b in enumerate(order):
            got[b].append(out[cu[i]:cu[i + 1]].cpu())

    for parts in ({0: 17, 1: 60, 2: 129}, {0: 2, 2: 1, 3: 1}, {0: 130, 2: 128, 3: 3}, {0: 1, 2: 2, 3: 5}, {2: 13}):
        step(parts)
    for b, n in enumerate(lens):
        o = torch.cat(got[b]).view(n, H, geo.vp)
        assert geo.vp == D or o[..., D:].abs().max() == 0
        close(o[..., :D].reshape(n, -1), want[b], dt, (shape, b))
    for part in (1, 3):         # slots nobody owns keep what they held
        assert (state.s[part] == 7.0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,B", [(6, 40, 300), (32, 64, 64), (1, 64, 1), (3, 128, 50)])
def test_decode_of_many_sequences(cuda_device, dtype, H, D, B):
    """More heads than CTAs, fresh and continued sequences and padding rows: the one-token kernels equal the scan."""
    geo = RecurrentGeometry(H, D, D, silu=False, gated=False)
    n, dev = H * geo.kp, cuda_device
    r, k, v, g, z = mix_case(geo, [B], 3, False)
    proj = torch.cat([padded(x, geo.kp) for x in (r, k, v, g)], 1).to(dtype).to(dev)
    mix = TimeMix(padded(z, geo.kp).to(dev), padded(rand(1, H, D, seed=8), geo.kp).view(-1).to(dev), padded(rand(1, H, D, seed=4), geo.kp).view(-1).to(dev))
    norm = padded(rand(1, H, D, seed=9) + 1.0, geo.kp).view(-1).to(dev)
    states = [RecurrentState.zeros(geo, B + 3, dev) for _ in range(2)]
    start = torch.zeros(B + 3, H, geo.kp, geo.vp)
    start[:, :, :D, :D] = rand(B + 3, H, D, D, seed=5)
    for s in states:
        s.s.copy_(start.view(B + 3, H, geo.kp, geo.tiles, 32).permute(0, 1, 3, 2, 4))
    slots = (torch.randperm(B, generator=torch.Generator().manual_seed(1)) + 2).int()
    lens = torch.where(torch.arange(B) % 5 == 3, 1, 20).int()
    if B > 2:
        slots[B // 2], slots[B - 1] = -1, -1
    slots, lens = slots.to(dev), lens.to(dev)
    o, outs = torch.zeros(B, n, device=dev), [torch.zeros(B, n, dtype=dtype, device=dev) for _ in range(2)]
    ops.recurrent_scan(proj, None, geo, None, None, None, 1.0, states[0], slots, torch.arange(B + 1, dtype=torch.int32, device=dev), lens, o, B, B, mix=mix)
    ops.gated_norm(o, norm, proj[:, 3 * n:], geo, 1e-5, outs[0], True, silu=True)
    ops.time_mix_decode(proj, geo, mix, states[1], slots, lens, norm, 1e-5, outs[1], B)
    ops.check_status()
    close(outs[1], outs[0].cpu(), dtype)
    close(states[1].s, states[0].s.cpu(), torch.float32)
    assert B <= 2 or outs[1][B - 1].abs().max() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("D", [40, 64, 128])
def test_many_chunks_and_sequences_at_once(cuda_device, D):
    """Sequences of one chunk and of many, fresh and continued: outputs and states equal the token-by-token form's."""
    geo = RecurrentGeometry(6, D, D, silu=False, gated=False)
    lens, done = [17, 128, 129, 900, 40, 2000], [0, 5, 0, 300, 64, 0]
    r, k, v, g, z = mix_case(geo, lens, 3, False)
    proj = torch.cat([padded(x, geo.kp) for x in (r, k, v, g)], 1).to(cuda_device)
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    T, n = cu[-1], 6 * geo.kp
    zeros = torch.zeros(n, device=cuda_device)
    norm = torch.ones(n, device=cuda_device)
    bonus = padded(rand(1, 6, D, seed=4), geo.kp).view(-1).to(cuda_device)
    states = [RecurrentState.zeros(geo, 8, cuda_device) for _ in range(2)]
    start = torch.zeros(8, 6, geo.kp, geo.vp)
    start[:, :, :D, :D] = rand(8, 6, D, D, seed=5)
    for s in states:
        s.s.copy_(start.view(8, 6, geo.kp, geo.tiles, 32).permute(0, 1, 3, 2, 4))
    slots, lens_t, cut = i32([7, 3, 0, 5, 1, 2], cuda_device), i32([a + b for a, b in zip(lens, done)], cuda_device), i32(cu, cuda_device)
    mix = TimeMix(padded(z, geo.kp).to(cuda_device), zeros, bonus)
    o, outs = torch.zeros(T, n, device=cuda_device), [torch.zeros(T, n, dtype=torch.bfloat16, device=cuda_device) for _ in range(2)]
    ops.recurrent_scan(proj, None, geo, None, None, None, 1.0, states[0], slots, cut, lens_t, o, T, 6, mix=mix)
    ops.gated_norm(o, norm, proj[:, 3 * n:], geo, 1e-5, outs[0], True, silu=True)
    table = ChunkTable.make(cu, 0, cuda_device)
    room = torch.empty(time_mix_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device=cuda_device)
    ops.time_mix_chunks(proj, geo, mix, states[1], slots, cut, lens_t, norm, 1e-5, outs[1], table, room)
    ops.check_status()
    close(outs[1], outs[0].cpu(), torch.bfloat16)
    close(states[1].s, states[0].s.cpu(), torch.float32)


# ------------------------------------------------------------------------------------------ experts, stream, token input
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("experts,top,ff,d,T", [(5, 2, 40, 56, 33), (1, 1, 8, 24, 3), (12, 12, 17, 30, 5), (64, 8, 192, 128, 300), (200, 1, 64, 64, 150)])
def test_experts_with_weighted_inputs(place, experts, top, ff, d, T):
    dev, dt = place
    width = -(-d // 8) * 8
    geo = ExpertsGeometry.make(experts, top, ff, width, None, dt, "sigmoid", False, True)
    w = {}
    for e in range(experts):
        for part, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
            w[f"m.e{e}.{part}"] = (rand(*shape, seed=7 * e + len(part)) * 2 / shape[1] ** 0.5).bfloat16()
    wgu = torch.zeros(experts * 2 * geo.ffp, width, dtype=dt, device=dev)
    wd = torch.zeros(experts * width, geo.ffp, dtype=dt, device=dev)
    ops.pack_experts(*([w[f"m.e{e}.{part}"].to(dev) for e in range(experts)] for part in ("gate", "up", "down")), geo, wgu, wd)
    scratch = ExpertsScratch(geo, T + 5, dt, torch.device(dev))
    for seed in (1, 2):
        h, z = rand(T, d, seed=seed, dtype=torch.bfloat16), rand(T, experts, seed=seed + 10)
        hp = torch.zeros(T, width, dtype=dt)
        hp[:, :d] = h
        y, p = ops.experts_forward(hp.to(dev), z.to(dev), geo, scratch, wgu, wd)
        assert p is None
        x = torch.zeros(T, width, device=dev)
        ops.stream_norm(x, d, experts=y, top=top, mult=0.6)
        wz, want = {k: v.double() for k, v in w.items()}, torch.zeros(T, d, dtype=torch.float64)
        best, pw = oracle.route(z.double(), top)
        for e in range(experts):
            t, j = (best == e).nonzero(as_tuple=True)
            want[t] += 0.6 * oracle.gated_unit(pw[t, j, None] * h[t].double(), wz, f"m.e{e}")
        close(x[:, :d], want, dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("d", [30, 200, 2048])
def test_stream_with_a_factor_and_a_normed_addend(place, d):
    dev, dt = place
    p = -(-d // 8) * 8

    def pad(x):
        out = torch.zeros(*x.shape[:-1], p)
        out[..., :d] = x
        return out.to(dev)

    x, y, s, sw, w = rand(6, d, seed=1), rand(6, d, seed=2), rand(6, d, seed=3) * 0.01, rand(d, seed=4), rand(d, seed=5)
    xs, h, copy = pad(x), torch.zeros(6, p, dtype=dt, device=dev), torch.zeros(6, p, dtype=dt, device=dev)
    ops.stream_norm(xs, d, y1=pad(y), side=pad(s), side_weight=pad(sw), mult=0.3, copy=copy, weight=pad(w), eps=1e-5, h=h)
    want = x.double() + 0.3 * (y.double() + oracle.rms(s.double(), 1e-5) * sw.double())
    close(xs[:, :d], want, torch.float32)
    close(copy[:, :d], want, dt)
    close(h[:, :d], oracle.rms(want, 1e-5) * w.double(), dt)


@pytest.mark.parametrize("place", PLACES)
def test_token_side_gate(place):
    dev, dt = place
    z, table, ids = rand(7, 24, seed=1) * 3, rand(11, 60, seed=2, dtype=torch.bfloat16), torch.tensor([3, 0, 10, 3, 1, 2, 9], dtype=torch.int32)
    out = torch.zeros(7, 24, dtype=dt, device=dev)
    ops.token_side(z.to(dev), ids.to(dev), table.to(dt).to(dev), 20, out, 20)
    close(out[:, :20], oracle.gelu_tanh(z[:, :20].double()) * table[ids.long(), 20:40].double(), dt)
    assert out[:, 20:].abs().max() == 0

"""The operations behind the Zamusun design one by one against the plain oracle (``zamusun_oracle.py``): CPU twins, and on a GPU
the kernels in bf16 and fp32. Recurrences and attention carry planted keys whose product with a late query stands out, so that
a lost state, a wrong chunk border or a missing sink cannot hide among many tokens."""

import pytest
import torch
import zamusun_oracle as oracle

from research_b200 import ops
from research_b200.ops.experts import ExpertsGeometry, ExpertsScratch
from research_b200.ops.keyvalue import KV_BLOCK, KeyValueGeometry
from research_b200.ops.recurrent import ChunkTable, RecurrentGeometry, RecurrentState, chunk_workspace

PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=pytest.mark.gpu),
          pytest.param(("cuda", torch.bfloat16), marks=pytest.mark.gpu)]


def close(got, want, dtype, what="", tol=None):
    tol = tol or (3e-5 if dtype == torch.float32 else 1.2e-2)
    err = (got.double().cpu() - want.double()).abs().max().item() / max(want.double().abs().max().item(), 1e-6)
    assert err < tol, (what, err)


def rand(*shape, seed, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


def i32(x, dev="cpu"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def padded(x, p):
    """[t, h, d] -> [t, h*p] with zero padding channels"""
    t, h, d = x.shape
    out = torch.zeros(t, h, p, dtype=x.dtype)
    out[..., :d] = x
    return out.view(t, h * p)


# ------------------------------------------------------------------------------------------ recurrences
SHAPES = [(3, 24, 20), (1, 7, 5), (2, 128, 128), (5, 64, 96), (2, 130, 40), (2, 250, 130), (2, 300, 33)]


def recurrent_case(geo, lens, seed, planted=True):
    """Packed q, k, v (rounded to bf16) and gate logits of several sequences. The planted key of a sequence is its second
    token's, found again by the queries of its last tokens."""
    T, H = sum(lens), geo.heads
    q, k, v = (rand(T, H, n, seed=seed + i, dtype=torch.bfloat16) for i, n in enumerate((geo.dim, geo.dim, geo.vdim)))
    k = k * 0.3
    small = torch.cat([rand(T, H, seed=seed + 4), rand(T, H, seed=seed + 5) + 5.0], 1)
    if planted:
        at = 0
        for n in lens:
            if n > 3:
                k[at + 1] = rand(H, geo.dim, seed=seed + 6, dtype=torch.bfloat16) * 4
                q[at + n - 2:at + n] = k[at + 1]
            at += n
    return q, k.bfloat16(), v, small


def recurrent_oracle(geo, q, k, v, small, decay, bi, bf, cap):
    q, k, v = q.double(), k.double(), v.double()
    if not geo.gated:
        return oracle.lightning_scan(q, k, v, decay.tolist())
    w = {"m.i": torch.eye(2 * geo.heads, dtype=torch.float64)[:geo.heads], "m.i.b": bi.double(),
         "m.f": torch.eye(2 * geo.heads, dtype=torch.float64)[geo.heads:], "m.f.b": bf.double()}
    i, f = oracle.mlstm_gates(small.double(), w, "m", cap)
    return oracle.mlstm_scan(q * geo.dim ** -0.5, k, v, i, f)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("shape", SHAPES)
def test_recurrences_in_portions_slots_and_batches(place, gated, shape):
    """Four sequences in dirty slots: portions that straddle chunk borders, down to two tokens, then single tokens."""
    dev, dt = place
    geo = RecurrentGeometry(*shape, silu=not gated, gated=gated)
    H, lens = geo.heads, [150, 60, 273, 9]
    decay = torch.linspace(0.5, 0.999, H) if H > 1 else torch.tensor([0.99])
    bi, bf, cap = rand(H, seed=50), rand(H, seed=51), 9.0
    data = [recurrent_case(geo, [n], 10 * b + 100) for b, n in enumerate(lens)]
    want = [recurrent_oracle(geo, *d, decay, bi, bf, cap) for d in data]
    state = RecurrentState.zeros(geo, 6, dev)
    for t in (state.s, state.n, state.m):
        t.fill_(7.0)
    slots = [4, 0, 5, 2]
    got = [[] for _ in lens]
    decay, bi, bf = decay.to(dev), bi.to(dev), bf.to(dev)

    def step(parts):
        """parts: {sequence: tokens}, sorted by length as the engine does"""
        order = sorted(parts, key=lambda b: parts[b])
        rows = {b: sum(len(x) for x in got[b]) for b in order}
        cols = [torch.cat([d[rows[b]:rows[b] + parts[b]] for b in order for d in (data[b][i],)]) for i in range(4)]
        proj = torch.cat([padded(cols[0], geo.kp), padded(cols[1], geo.kp), padded(cols[2], geo.vp), padded(cols[2], geo.vp)], 1).to(dt).to(dev)
        T = proj.shape[0]
        cu = [0]
        for b in order:
            cu.append(cu[-1] + parts[b])
        out = torch.full((T, H * geo.vp), 9.0, device=dev)
        small = cols[3].to(dev) if gated else None
        a = (proj, small, geo, decay, bi, bf, cap, state, i32([slots[b] for b in order], dev))
        tail = (i32(cu, dev), i32([rows[b] + parts[b] for b in order], dev), out)
        single = next((i for i, b in enumerate(order) if parts[b] > 1), len(order))
        short = next((i for i, b in enumerate(order) if parts[b] > 16), len(order)) if dt == torch.bfloat16 and geo.kp <= 256 else len(order)
        if single:
            ops.recurrent_scan(*a, None, *tail[1:], single, single)
        if short > single:
            ops.recurrent_scan(*a, *tail, cu[short], short, single)
        if short < len(order):
            table = ChunkTable.make(cu, short, dev)
            ops.recurrent_chunks(*a, *tail, table, torch.empty(chunk_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device=dev))
        for i, b in enumerate(order):
            got[b].append(out[cu[i]:cu[i + 1]].cpu())

    for parts in ({0: 17, 1: 60, 2: 129}, {0: 2, 2: 1, 3: 1}, {0: 130, 2: 128, 3: 3}, {0: 1, 2: 2, 3: 5}, {2: 13}):
        step(parts)
    for b, n in enumerate(lens):
        o = torch.cat(got[b]).view(n, H, geo.vp)
        assert o[..., geo.vdim:].abs().max() == 0 if geo.vp > geo.vdim else True
        close(o[..., :geo.vdim], want[b], dt, (shape, b))
    for part in (1, 3):         # slots nobody owns keep what they held
        assert (state.s[part] == 7.0).all() and (state.m[part] == 7.0).all()


@pytest.mark.gpu
def test_many_chunks_and_sequences_at_once(cuda_device):
    """More work units than CTAs, sequences of one chunk and of many, fresh and continued."""
    geo = RecurrentGeometry(6, 64, 192, silu=False, gated=True)
    lens, done = [17, 128, 129, 900, 40, 2000], [0, 5, 0, 300, 64, 0]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    T, H = cu[-1], 6
    q, k, v, small = recurrent_case(geo, lens, 3)
    proj = torch.cat([padded(q, 64), padded(k, 64), padded(v, 192), padded(v, 192)], 1).to(cuda_device)
    bi, bf = rand(H, seed=1).to(cuda_device), rand(H, seed=2).to(cuda_device)
    states = [RecurrentState.zeros(geo, 8, cuda_device) for _ in range(2)]
    for s in states:
        s.s.copy_(rand(*s.s.shape, seed=4))
        s.n.copy_(rand(8, H, 1, 64, seed=5).expand_as(s.n))
        s.m.copy_(rand(8, H, 1, seed=6).expand_as(s.m))
    slots, lens_t = i32([7, 3, 0, 5, 1, 2], cuda_device), i32([a + b for a, b in zip(lens, done)], cuda_device)
    outs = []
    for s, chunked in zip(states, (False, True)):
        out = torch.zeros(T, H * 192, device=cuda_device)
        a = (proj, small.to(cuda_device), geo, None, bi, bf, 12.0, s, slots, i32(cu, cuda_device), lens_t, out)
        if chunked:
            table = ChunkTable.make(cu, 0, cuda_device)
            ops.recurrent_chunks(*a, table, torch.empty(chunk_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device=cuda_device))
        else:
            ops.recurrent_scan(*a, T, 6)
        outs.append(out)
    close(outs[1], outs[0].cpu(), torch.bfloat16)
    close(states[1].s, states[0].s.cpu(), torch.float32)
    close(states[1].n, states[0].n.cpu(), torch.float32)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("per_head", [True, False])
@pytest.mark.parametrize("shape", [(3, 8, 20), (9, 8, 128), (1, 8, 3)])
def test_norm_and_gate(place, per_head, shape):
    dev, dt = place
    geo = RecurrentGeometry(*shape, silu=False, gated=True)
    H, V, T = geo.heads, geo.vdim, 5
    o, w, g = rand(T, H, V, seed=1) * 3, rand(H * V, seed=2) + 1, rand(T, H, V, seed=3, dtype=torch.bfloat16).float()
    normed = oracle.rms(o.double(), 1e-4).view(T, H * V) if per_head else oracle.rms(o.double().view(T, H * V), 1e-4)
    want = normed * w.double() * torch.sigmoid(g.double().view(T, H * V))
    out = torch.zeros(T, H * geo.vp, dtype=dt, device=dev)
    gate = torch.cat([torch.ones(T, 8), padded(g, geo.vp)], 1).to(dt).to(dev)[:, 8:]
    ops.gated_norm(padded(o, geo.vp).to(dev), padded(w.view(1, H, V), geo.vp).view(-1).to(dev), gate, geo, 1e-4, out, per_head)
    close(out.view(T, H, geo.vp)[..., :V].reshape(T, H * V), want, dt)


# ------------------------------------------------------------------------------------------ attention whose values are its keys
HEADS = [(6, 2, 24), (1, 1, 7), (8, 1, 128), (40, 2, 64), (4, 4, 136), (3, 1, 300)]


def kv_oracle(q, k, gate, sink, scale, coef, every):
    """The oracle's attention on given projections: identity matrices stand for the projections."""
    t, H, D = q.shape
    G = k.shape[1]
    h = torch.cat([q.reshape(t, -1), k.reshape(t, -1), gate.reshape(t, -1)], 1).double()
    eye = torch.eye(h.shape[1], dtype=torch.float64)
    w = {"m.q": eye[:H * D], "m.k": eye[H * D:(H + G) * D], "m.g": eye[(H + G) * D:], "m.o": torch.eye(H * D, dtype=torch.float64), "m.sink": sink.double()}
    return oracle.attention(h, w, "m", {"heads": H, "kv_heads": G, "dim": D, "scale": scale, "q_temp": {"coef": coef, "every": every}}, 0.0)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", HEADS)
@pytest.mark.parametrize("splits", [1, 3])
def test_keys_as_values_attention_finds_planted_keys(place, shape, splits):
    """Scattered blocks, prompts and single tokens together; a key of every sequence stands out for its late queries: the first
    one, those at a block's borders, the token itself."""
    dev, dt = place
    H, G, D = shape
    geo = KeyValueGeometry(H, G, D)
    scale, coef, every = 1.5 * D ** -0.5, 0.3, 7
    lens, done = [70, 300, 33, 130, 257], [69, 299, 32, 0, 100]
    plant = [0, 15, 16, 31, 127]
    sink = rand(H, seed=9) + 1.0
    nb = 80
    cache = torch.zeros(nb, G, KV_BLOCK, geo.dp, dtype=dt, device=dev)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(1)).tolist()
    tables, rows, wants, meta, at = torch.zeros(5, 24, dtype=torch.int32), [], [], [], 0
    for b, (L, d0) in enumerate(zip(lens, done)):
        q, k, gate = (rand(L, n, D, seed=30 + 3 * b + i, dtype=torch.bfloat16) for i, n in enumerate((H, G, H)))
        k[plant[b]] = 2.0 * rand(G, D, seed=70 + b).sign().bfloat16()
        q[L - 3:] = k[plant[b]].repeat_interleave(H // G, 0)
        nblk = -(-L // KV_BLOCK)
        tables[b, :nblk] = torch.tensor(perm[at:at + nblk])
        at += nblk
        proj = torch.cat([padded(q, geo.dp), padded(k, geo.dp), padded(gate, geo.dp)], 1)
        pos = torch.arange(L)
        slot = tables[b, pos // KV_BLOCK] * KV_BLOCK + pos % KV_BLOCK
        wants.append(kv_oracle(q, k, gate, sink, scale, coef, every)[d0:])
        meta.append((proj, pos.int(), slot.int(), d0))
    sinks = sink.to(dev)
    for proj, pos, slot, d0 in meta:                    # what is cached already
        if d0:
            ops.kv_append(proj[:d0].to(dt).to(dev), geo, pos[:d0].to(dev), slot[:d0].to(dev), coef, every, cache)
    new = torch.cat([p[d0:] for p, _, _, d0 in meta]).to(dt).to(dev)
    ops.kv_append(new, geo, torch.cat([p[d0:] for _, p, _, d0 in meta]).to(dev), torch.cat([s[d0:] for _, _, s, d0 in meta]).to(dev), coef, every, cache)
    cu = [0]
    for L, d0 in zip(lens, done):
        cu.append(cu[-1] + L - d0)
    out = torch.full((cu[-1], H * geo.dp), 5.0, dtype=dt, device=dev)
    ws = torch.zeros(ops.kv_workspace(geo, 5, splits), device=dev)
    ops.kv_attention(new, geo, cache, tables.to(dev), i32(cu, dev), i32(lens, dev), sinks, out, scale=scale, rows=cu[-1], max_q=157, n_single=3,
                     workspace=ws, splits=splits)
    for b in range(5):
        got = out[cu[b]:cu[b + 1]].view(-1, H, geo.dp)[..., :D].reshape(-1, H * D)
        close(got, wants[b], dt, (shape, b))
    # the same single tokens as a decode batch with a padding row
    single = torch.cat([new[:3], new[:1]])
    dec = torch.full((4, H * geo.dp), 5.0, dtype=dt, device=dev)
    ops.kv_attention(single, geo, cache, torch.cat([tables[:3], tables[:1]]).to(dev), None, i32(lens[:3] + [0], dev), sinks, dec, scale=scale, rows=4, max_q=1,
                     n_single=4, workspace=ws, splits=splits)
    close(dec[:3], out[:3].cpu(), dt)
    assert dec[3].abs().max() == 0


@pytest.mark.parametrize("place", PLACES)
def test_query_temperature_steps_and_skipped_rows(place):
    dev, dt = place
    geo = KeyValueGeometry(2, 1, 8)
    pos = torch.tensor([0, 5, 6, 7, 13, 1000, 3], dtype=torch.int32)
    proj = rand(7, geo.proj, seed=2, dtype=torch.bfloat16)
    cache = torch.full((4, 1, KV_BLOCK, 64), 3.0, dtype=dt, device=dev)
    got = proj.to(dt).to(dev)
    ops.kv_append(got, geo, pos.to(dev), i32([0, 17, 63, 16, 5, 40, -1], dev), 0.5, 7, cache)
    want = proj[:, :128].double() * oracle.query_temperature(pos, 0.5, 7)[:, None]
    close(got[:, :128], want, dt)
    assert torch.equal(got[:, 128:].cpu(), proj[:, 128:].to(dt))
    assert torch.equal(cache[1, 0, 1].cpu(), proj[1, 128:192].to(dt)) and torch.equal(cache[3, 0, 15].cpu(), proj[2, 128:192].to(dt))
    assert int((cache == 3.0).all(-1).sum()) == 64 - 6


# ------------------------------------------------------------------------------------------ experts, stream, epilogues
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("experts,top,ff,d,T", [(5, 2, 40, 56, 33), (1, 1, 8, 24, 3), (12, 12, 17, 30, 5), (64, 8, 192, 128, 300), (200, 3, 64, 64, 150)])
def test_routed_experts(place, experts, top, ff, d, T):
    """Twice with one scratch: the histogram is left empty; some experts get every token, some none."""
    dev, dt = place
    width = -(-d // 8) * 8
    geo = ExpertsGeometry.make(experts, top, ff, width, 1.25, dt)
    w = {}
    for e in range(experts):
        for part, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
            w[f"m.e{e}.{part}"] = (rand(*shape, seed=7 * e + len(part)) * 2 / shape[1] ** 0.5).bfloat16()
    wgu = torch.zeros(experts * 2 * geo.ffp, width, dtype=dt, device=dev)
    wd = torch.zeros(experts * width, geo.ffp, dtype=dt, device=dev)
    ops.pack_experts(*([w[f"m.e{e}.{part}"].to(dev) for e in range(experts)] for part in ("gate", "up", "down")), geo, wgu, wd)
    scratch = ExpertsScratch(geo, T + 5, dt, torch.device(dev))
    for seed in (1, 2):
        h = rand(T, d, seed=seed, dtype=torch.bfloat16)
        z = rand(T, experts, seed=seed + 10)
        z[:, 0] += 6.0                                   # everyone's first choice
        logits = torch.zeros(T, experts + 3)
        logits[:, :experts], logits[:, experts:] = z, 99.0
        hp = torch.zeros(T, width, dtype=dt)
        hp[:, :d] = h
        y, p = ops.experts_forward(hp.to(dev), logits.to(dev)[:, :experts] if experts % 4 else logits.to(dev), geo, scratch, wgu, wd)
        x = torch.zeros(T, width, device=dev)
        ops.stream_norm(x, d, experts=y, expert_weights=p)
        wz = {k: v.double() for k, v in w.items()}
        want = torch.zeros(T, d, dtype=torch.float64)
        best, pw = oracle.route(z.double(), top)
        for e in range(experts):
            t, j = (best == e).nonzero(as_tuple=True)
            want[t] += pw[t, j, None] * oracle.expert(h[t].double(), wz, f"m.e{e}", 1.25)
        close(x[:, :d], want, dt)
        assert width == d or x[:, d:].abs().max() == 0


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("d", [30, 200, 2048])
def test_stream_update_and_norm(place, d):
    dev, dt = place
    p = -(-d // 8) * 8

    def pad(x):
        out = torch.zeros(*x.shape[:-1], p)
        out[..., :d] = x
        return out

    x, y1, y2, e, w = rand(6, d, seed=1), rand(6, d, seed=2), rand(6, d, seed=3), rand(18, d, seed=4, dtype=torch.bfloat16), rand(d, seed=5)
    ew = torch.rand(6, 3)
    want = (x + y1 + y2).double() + (e.double().view(6, 3, d) * ew.double()[..., None]).sum(1)
    xs = pad(x).to(dev)
    h, copy = torch.zeros(6, p, dtype=dt, device=dev), torch.zeros(6, 2 * p, dtype=dt, device=dev)
    ops.stream_norm(xs, d, y1=pad(y1).to(dev), y2=pad(y2).to(dev), experts=pad(e.float()).to(dt).to(dev), expert_weights=ew.to(dev),
                    copy=copy[:, :p], weight=pad(1 + w).to(dev), eps=1e-3, h=h)
    close(xs[:, :d], want, torch.float32)
    close(copy[:, :d], want, dt)
    assert copy[:, p:].abs().max() == 0
    close(h[:, :d], oracle.rms(want, 1e-3) * (1 + w.double()), dt)
    rows = torch.tensor([5, 0, 0], dtype=torch.int32)
    out = torch.zeros(3, p, dtype=dt, device=dev)
    ops.stream_norm(xs, d, weight=pad(1 + w).to(dev), eps=1e-3, h=out, rows=rows.to(dev))
    close(out[:, :d], oracle.rms(want, 1e-3)[rows.long()] * (1 + w.double()), dt)
    ids = torch.tensor([3, 0, 2], dtype=torch.int32)
    table = pad(rand(4, d, seed=6)).to(dt)
    xs, both = torch.zeros(3, p, device=dev), torch.zeros(3, 2 * p, dtype=dt, device=dev)
    ops.stream_embed(ids.to(dev), table.to(dev), d, xs, both[:, :p], both[:, p:])
    assert torch.equal(xs.cpu(), table[ids.long()].float()) and torch.equal(both[:, p:].cpu(), table[ids.long()]) and torch.equal(both[:, :p], both[:, p:])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("M,cols,K,silu,tail", [(3, 96, 72, 64, 8), (130, 704, 256, 192, 24), (256, 2112, 2048, 1536, 64), (1024, 4160, 512, 4096, 72),
                                                (1, 224, 4096, 0, 40)])
def test_projection_with_activated_columns_and_a_narrow_tail(place, M, cols, K, silu, tail):
    """One-CTA, split-K and two-CTA products alike."""
    dev, dt = place
    N = cols + tail
    a, b, bias = rand(M, K, seed=1, dtype=torch.bfloat16), (rand(N, K, seed=2) / K ** 0.5).bfloat16(), rand(N, seed=3, dtype=torch.bfloat16)
    want = a.double() @ b.double().T + bias.double()
    rest = want[:, cols:].clone()
    want[:, :silu] = oracle.silu(want[:, :silu])
    t = torch.zeros(M, tail, device=dev)
    out = torch.zeros(M, cols, dtype=dt, device=dev)
    ops.gemm(a.to(dt).to(dev), b.to(dt).to(dev), bias=bias.to(dt).to(dev), out=out, silu_cols=silu, tail=t)
    close(out, want[:, :cols], dt)
    close(t, rest, torch.float32)

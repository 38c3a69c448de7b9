"""The operations of the Lulezen design one by one against the plain oracle (``lulezen_oracle.py``): CPU twins, and on a GPU
the kernels in bf16 and fp32. Attention inputs carry planted keys whose score stands out, just inside and just outside the
window, at block borders and far away, so that a wrong edge, block or sink cannot hide among many keys."""

import math

import lulezen_oracle as oracle
import pytest
import torch

from research_b200 import ops
from research_b200.ops.gemm import gemm_f32_batched
from research_b200.ops.latent import LatentGeometry

PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=pytest.mark.gpu),
          pytest.param(("cuda", torch.bfloat16), marks=pytest.mark.gpu)]
GEOMETRIES = [LatentGeometry(5, 40, 12, 6, 24, 72, 44), LatentGeometry(1, 7, 2, 1, 5, 9, 10), LatentGeometry(16, 128, 64, 32, 128, 512, 200),
              LatentGeometry(40, 64, 32, 16, 64, 250, 64), LatentGeometry(3, 16, 8, 2, 16, 600, 24),
              LatentGeometry(20, 16, 64, 32, 16, 1024, 24)]


def close(got, want, dtype, what=""):
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    err = (got.double().cpu() - want.double()).abs().max().item() / max(want.double().abs().max().item(), 1e-6)
    assert err < tol, (what, err)


def rand(*shape, seed, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


# ------------------------------------------------------------------------------------------ norms, unit, cap, products
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("d", [30, 513, 2048])
def test_layer_norm_on_the_residual_and_final_norm(place, d):
    dev, dt = place
    y, x, w, b = rand(9, d + 2, seed=1) * 3 + 2, rand(9, d, seed=2), rand(d, seed=3), rand(d, seed=4)
    want = x.double() + oracle.layer_norm(y[:, :d].double(), w.double(), b.double(), 1e-3)
    xg, xb = x.clone().to(dev), torch.zeros(9, d + 2, dtype=dt, device=dev)
    ops.layernorm_residual(y.to(dev), w.to(dev), b.to(dev), 1e-3, xg, xb)
    close(xg, want, torch.float32)
    close(xb[:, :d], want, dt)
    assert xb[:, d:].abs().max() == 0
    rows = torch.tensor([8, 8, 0, 3], dtype=torch.int32)
    out = torch.zeros(4, d, dtype=dt, device=dev)
    ops.layernorm_rows(x.to(dev), w.to(dev), b.to(dev), 1e-3, out, rows.to(dev))
    close(out, oracle.layer_norm(x.double()[rows.long()], w.double(), b.double(), 1e-3), dt)


@pytest.mark.parametrize("place", PLACES)
def test_clamped_unit_and_soft_cap(place):
    dev, dt = place
    gu = (rand(17, 2 * 48, seed=5) * 4).to(dt)
    eye = torch.eye(48, dtype=torch.float64)
    for limit in (0.5, 2.0, 7.0):
        w = {"m.gate": torch.eye(96, dtype=torch.float64)[:48], "m.up": torch.eye(96, dtype=torch.float64)[48:], "m.down": eye}
        close(ops.clamped_glu(gu.to(dev), limit), oracle.clamped_swiglu(gu.double(), w, "m", limit), dt)
    x = rand(11, 37, seed=6) * 30
    close(ops.softcap(x.clone().to(dev), 12.0), 12.0 * torch.tanh(x.double() / 12.0), torch.float32)


@pytest.mark.gpu
def test_gemm_epilogues_and_f32_products(cuda_device):
    a, g, u = rand(130, 200, seed=7, dtype=torch.bfloat16), rand(256, 200, seed=8, dtype=torch.bfloat16), rand(256, 200, seed=9, dtype=torch.bfloat16)
    w = {"m.gate": g.double() / 8, "m.up": u.double() / 8, "m.down": torch.eye(256, dtype=torch.float64)}
    packed = ops.interleave_gate_up((g / 8).to(cuda_device), (u / 8).to(cuda_device), 256)
    got = ops.gemm(a.to(cuda_device), packed, bn=256, swiglu=True, glu_limit=1.5)
    close(got, oracle.clamped_swiglu(a.double(), w, "m", 1.5), torch.bfloat16)
    z = a.double() @ g.double().T
    close(ops.gemm(a.to(cuda_device), g.to(cuda_device), out_f32=True, softcap=25.0), 25.0 * torch.tanh(z / 25.0), torch.float32)
    x, y = rand(3, 70, 37, seed=10), rand(3, 90, 37, seed=11)
    out = torch.zeros(3, 70, 90, device=cuda_device)
    gemm_f32_batched(x.to(cuda_device), y.to(cuda_device), out, 70, 90, 37, 3, (37, 37, 90), (70 * 37, 90 * 37, 70 * 90))
    close(out, x.double() @ y.double().transpose(1, 2), torch.float32)
    yt = y.transpose(1, 2).contiguous()
    gemm_f32_batched(x.to(cuda_device), yt.to(cuda_device), out, 70, 90, 37, 3, (37, 90, 90), (70 * 37, 90 * 37, 70 * 90), b_kn=True)
    close(out, x.double() @ y.double().transpose(1, 2), torch.float32)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("geo", GEOMETRIES)
def test_append_query_and_head_products(place, geo):
    dev, dt = place
    T, S, eps = 11, 24, 1e-4
    H, q0, k0, r0 = geo.heads, geo.q_rank, geo.q_rank + geo.kv_rank, geo.q_rank + geo.kv_rank + geo.rot_dim
    pos = torch.tensor([0, 1, 2, 15, 16, 17, 500, 900, 901, 31, 32], dtype=torch.int32)
    slots = torch.tensor([3, 16, 17, 47, 0, -1, 63, 20, 21, 5, 33], dtype=torch.int32)
    base = 700.0
    table = ops.rope_table(1024, 2 * geo.rot_pairs, base, exact=True)
    proj = rand(T, geo.proj, seed=20)
    qn_w, kn_w = 1 + 0.3 * rand(geo.q_rank, seed=21), 1 + 0.3 * rand(geo.kv_rank, seed=22)
    cache = torch.zeros(4, 16, geo.cw, dtype=dt, device=dev)
    cq, gate = torch.zeros(T, geo.qp, dtype=dt, device=dev), torch.zeros(T, H, device=dev)
    ops.latent_append(proj.to(dev), geo, qn_w.to(dev), kn_w.to(dev), eps, pos.to(dev), slots.to(dev), table.to(dev), cache, cq, gate)
    p = proj.double()
    close(cq[:, :q0], oracle.rms(p[:, :q0], qn_w.double(), eps), dt, "query latent")
    close(gate, torch.sigmoid(p[:, r0:r0 + H]), torch.float32, "gate")
    want = torch.zeros(64, geo.cw, dtype=torch.float64)
    ok = slots >= 0
    want[slots[ok].long(), :geo.kv_rank] = oracle.rms(p[ok][:, q0:k0], kn_w.double(), eps)
    want[slots[ok].long(), geo.rw:geo.rw + geo.rot_dim] = oracle.rotate(p[ok][:, k0:r0], pos[ok], 2 * geo.rot_pairs, base)
    close(cache.view(64, geo.cw), want, dt, "cache rows")

    q = rand(T, H, geo.dp + geo.rp, seed=23).to(dt)
    turned = oracle.rotate(q[..., geo.dp:geo.dp + geo.rot_dim].double(), pos, 2 * geo.rot_pairs, base)
    n = 7
    qg, qn = q.clone().to(dev), torch.zeros(H, S, geo.dp, dtype=dt, device=dev)
    qa = torch.zeros(H, S, geo.cw, dtype=dt, device=dev)
    ops.latent_query(qg.view(T, -1), geo, pos.to(dev), table.to(dev), n, qn, qa)
    assert torch.equal(qn[:, :n].cpu(), q[:n, :, :geo.dp].transpose(0, 1)) and qn[:, n:].abs().max() == 0
    close(qa[:, :n, geo.rw:geo.rw + geo.rot_dim], turned[:n].transpose(0, 1), dt, "rotated, short")
    close(qg[n:, :, geo.dp:geo.dp + geo.rot_dim], turned[n:], dt, "rotated in place")
    assert torch.equal(qg[n:, :, :geo.dp].cpu(), q[n:, :, :geo.dp])

    wuk, wuv = rand(H * geo.dp, geo.rw, seed=24).to(dt), rand(H * geo.vp, geo.rw, seed=25).to(dt)
    ops.head_gemm_absorb(qn, wuk.to(dev), qa, n)
    close(qa[:, :n, :geo.rw], torch.einsum("thd,hdr->htr", q[:n, :, :geo.dp].double(), wuk.double().view(H, geo.dp, geo.rw)), dt, "absorb")
    assert qa[:, n:].abs().max() == 0
    ol = rand(H, S, geo.rw, seed=26).to(dt)
    out = torch.zeros(T, H * geo.vp, dtype=dt, device=dev)
    ops.head_gemm_expand(ol.to(dev), wuv.to(dev), out, n)
    close(out[:n], torch.einsum("htr,hvr->thv", ol[:, :n].double(), wuv.double().view(H, geo.vp, geo.rw)).reshape(n, -1), dt, "expand")
    assert out[n:].abs().max() == 0


# ------------------------------------------------------------------------------------------ attention
def plain_attention(q, keys, values, n_new, window, scale, sink, gate):
    """q [t, h, c], keys [k, c] or [k, h, c], values likewise; the t queries are the last of the k positions."""
    k = keys.shape[0]
    s = (torch.einsum("thc,kc->htk", q, keys) if keys.dim() == 2 else torch.einsum("thc,khc->htk", q, keys)) * scale
    s = s.masked_fill(~oracle.visible(k, window)[k - n_new:][None], -math.inf)
    p = oracle.softmax_with_sink(s, sink)
    o = torch.einsum("htk,kc->thc", p, values) if values.dim() == 2 else torch.einsum("htk,khc->thc", p, values)
    return o * gate[..., None]


def plant(q, keys, spots, scale, height=6.0):
    """Make the key at every spot answer the query (t, head) with a score of ``height``: the query gets a private channel-like
    direction by aligning the key with it. q [t, h, c] (one sequence), keys [k, c]."""
    for t, h, key in spots:
        v = q[t, h]
        keys[key] = v * (height / (scale * float(v @ v)))


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("geo", GEOMETRIES)
@pytest.mark.parametrize("decode", [False, True])
def test_attention_on_cached_latents(place, geo, decode):
    dev, dt = place
    H, S, window = geo.heads, 48, 70
    lens = [1, 16, 37, 150, 333, 70, 71]
    new = [1] * 7 if decode else [1, 5, 16, 2, 13, 1, 3]
    T, scale = sum(new), 1.0 / math.sqrt(geo.cw)
    blocks = torch.randperm(64, generator=torch.Generator().manual_seed(1)).int()
    cache = torch.zeros(64, 16, geo.cw)
    bt, at = torch.zeros(len(lens), 24, dtype=torch.int32), 0
    qa = torch.zeros(H, S, geo.cw)
    sink, gate = rand(H, seed=3) + 1, torch.sigmoid(rand(T, H, seed=4))
    rows, t0 = [], 0
    for b, (L, n) in enumerate(zip(lens, new)):
        keys = torch.zeros(L, geo.cw)
        keys[:, :geo.kv_rank] = rand(L, geo.kv_rank, seed=10 + b)
        keys[:, geo.rw:geo.rw + geo.rot_dim] = rand(L, geo.rot_dim, seed=30 + b)
        q = torch.zeros(n, H, geo.cw)
        q[..., :geo.kv_rank] = rand(n, H, geo.kv_rank, seed=50 + b)
        q[..., geo.rw:geo.rw + geo.rot_dim] = rand(n, H, geo.rot_dim, seed=70 + b)
        pos = L - 1
        # oldest visible key, the one before it, block borders, the first token, the query itself
        spots = [(n - 1, h % H, k) for h, k in enumerate((pos - window + 1, pos - window, pos, 16 * (pos // 16), 16 * (pos // 16) - 1, 0)) if 0 <= k < L]
        plant(q, keys, spots, scale)
        q, keys = q.to(dt), keys.to(dt)
        qa[:, t0:t0 + n] = q.transpose(0, 1).float()
        nb = -(-L // 16)
        bt[b, :nb] = blocks[at:at + nb]
        at += nb
        flat = cache.view(-1, geo.cw)
        for k in range(L):
            flat[int(bt[b, k // 16]) * 16 + k % 16, :geo.cw] = keys[k].float()
        rows.append(plain_attention(q.double(), keys.double(), keys[:, :geo.rw].double(), n, window, scale, sink.double(), gate[t0:t0 + n].double()))
        t0 += n
    want = torch.cat(rows).transpose(0, 1)
    cu = None if decode else torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32).to(dev)
    sl = torch.tensor(lens, dtype=torch.int32).to(dev)
    out = torch.zeros(H, S, geo.rw, dtype=dt, device=dev)
    plan = ws = None
    if dev == "cuda" and dt == torch.bfloat16:
        plan = torch.zeros(ops.latent_units(len(lens), H, max(new)) + 1, dtype=torch.int32, device=dev)
        ops.latent_plan(cu, sl, geo, max(new), window, plan)
        ws = ops.latent_workspace([geo], dev)
    ops.latent_attention(qa.to(dt).to(dev), cache.to(dt).to(dev), geo, bt.to(dev), cu, sl, sink.to(dev), gate.to(dev), out, scale=scale,
                         window=window, rows=T, max_q=max(new), plan=plan, workspace=ws)
    close(out[:, :T], want, dt)
    assert out[:, T:].abs().max() == 0


@pytest.mark.gpu
def test_attention_shares_cut_anywhere(cuda_device):
    """Many batch shapes, so that the CTAs' equal shares cut units at all kinds of places; padding rows stay harmless."""
    geo, dt = LatentGeometry(6, 32, 16, 8, 32, 100, 64), torch.bfloat16
    ws = ops.latent_workspace([geo], cuda_device)
    for seed, (B, longest, window) in enumerate([(1, 1000, 5000), (2, 700, 333), (37, 400, 100), (150, 90, 64), (300, 50, 17)]):
        g = torch.Generator().manual_seed(seed)
        lens = torch.randint(0, longest + 1, (B,), generator=g).int()
        lens[0] = longest
        nb = -(-longest // 16)
        bt = torch.randperm(B * nb, generator=g).int().view(B, nb)
        cache = rand(B * nb, 16, geo.cw, seed=seed, dtype=dt)
        cache[..., geo.kv_rank:geo.rw] = 0
        cache[..., geo.rw + geo.rot_dim:geo.cw] = 0
        qa, sink, gate = rand(geo.heads, B, geo.cw, seed=seed + 9, dtype=dt), rand(geo.heads, seed=1), torch.sigmoid(rand(B, geo.heads, seed=2))
        plan = torch.zeros(B + 1, dtype=torch.int32, device=cuda_device)
        sl = lens.to(cuda_device)
        ops.latent_plan(None, sl, geo, 1, window, plan)
        out = torch.zeros(geo.heads, B, geo.rw, dtype=dt, device=cuda_device)
        ops.latent_attention(qa.to(cuda_device), cache.to(cuda_device), geo, bt.to(cuda_device), None, sl, sink.to(cuda_device),
                             gate.to(cuda_device), out, scale=0.1, window=window, rows=B, max_q=1, plan=plan, workspace=ws)
        for b in range(B):
            L = int(lens[b])
            if L == 0:
                continue
            k = torch.arange(L)
            keys = cache.view(-1, geo.cw)[bt[b, k // 16].long() * 16 + k % 16, :geo.cw].double()
            want = plain_attention(qa[:, b][None].double(), keys, keys[:, :geo.rw], 1, window, 0.1, sink.double(), gate[b:b + 1].double())
            close(out[:, b], want[0], dt, (B, b, L))


@pytest.mark.gpu
@pytest.mark.parametrize("heads", [3, 20])
def test_attention_is_repeatable(cuda_device, heads):
    """Hand-offs between the kernel's warps: short sequences (few tiles per CTA, cut units) give the same bits every time."""
    geo, B = LatentGeometry(heads, 24, 8, 4, 20, 40, 36), 5
    g = torch.Generator().manual_seed(4)
    bt = torch.randperm(B * 10, generator=g).int().view(B, 10).to(cuda_device)
    sl = torch.tensor([97, 120, 33, 150, 49], dtype=torch.int32, device=cuda_device)
    cache, qa = rand(B * 10, 16, geo.cw, seed=1, dtype=torch.bfloat16).to(cuda_device), (3 * rand(heads, B, geo.cw, seed=2)).bfloat16().to(cuda_device)
    sink, gate = rand(heads, seed=3).to(cuda_device), torch.sigmoid(rand(B, heads, seed=4)).to(cuda_device)
    plan = torch.zeros(ops.latent_units(B, heads, 1) + 1, dtype=torch.int32, device=cuda_device)
    ops.latent_plan(None, sl, geo, 1, 1000, plan)
    ws, first = ops.latent_workspace([geo], cuda_device), None
    for _ in range(300):
        out = torch.zeros(heads, B, geo.rw, dtype=torch.bfloat16, device=cuda_device)
        ops.latent_attention(qa, cache, geo, bt, None, sl, sink, gate, out, scale=0.3, window=1000, rows=B, max_q=1, plan=plan, workspace=ws)
        first = out if first is None else first
        assert torch.equal(out, first)


@pytest.mark.parametrize("place", [PLACES[0], PLACES[2]])
@pytest.mark.parametrize("geo", [LatentGeometry(4, 40, 12, 6, 24, 72, 44), LatentGeometry(2, 128, 64, 32, 128, 96, 64),
                                 LatentGeometry(3, 100, 64, 32, 50, 64, 64), LatentGeometry(3, 50, 40, 16, 128, 80, 64)])
@pytest.mark.parametrize("window", [1, 17, 128, 129, 1000])
def test_expanded_attention_and_gather(place, geo, window):
    """Long portions: cached rows gathered, multiplied out, attended; planted keys at and beyond the window's edge."""
    dev, dt = place
    H, scale = geo.heads, 0.15
    new, before, lead = [17, 128, 129, 300], [0, 63, 5, 410], 3
    T = lead + sum(new)
    cu_q = torch.tensor([lead] + [lead + int(x) for x in torch.tensor(new).cumsum(0)], dtype=torch.int32)
    lens = [n + p for n, p in zip(new, before)]
    lo = [max(0, p - window + 1) for p in before]
    cu_k = torch.tensor([0] + list(torch.tensor([L - x for L, x in zip(lens, lo)]).cumsum(0)), dtype=torch.int32)
    S = int(cu_k[-1])
    wuk, wuv = (rand(H * geo.dp, geo.rw, seed=1) / 6).to(dt), (rand(H * geo.vp, geo.rw, seed=2) / 6).to(dt)
    q = torch.zeros(T, H, geo.dp + geo.rp)
    q[..., :geo.dim], q[..., geo.dp:geo.dp + geo.rot_dim] = rand(T, H, geo.dim, seed=3), rand(T, H, geo.rot_dim, seed=4)
    q = q.to(dt)
    sink, gate = rand(H, seed=5) * 2, torch.sigmoid(rand(T, H, seed=6))
    cache, bt, at, rows = torch.zeros(160, 16, geo.cw), torch.zeros(4, 48, dtype=torch.int32), 0, []
    perm = torch.randperm(160, generator=torch.Generator().manual_seed(7)).int()
    for b, L in enumerate(lens):
        c = torch.zeros(L, geo.cw)
        c[:, :geo.kv_rank], c[:, geo.rw:geo.rw + geo.rot_dim] = rand(L, geo.kv_rank, seed=20 + b), rand(L, geo.rot_dim, seed=40 + b)
        t_last, pos = new[b] - 1, L - 1
        for h, k in enumerate((pos - window + 1, pos - window, pos - 128, 0)):      # planted in the rotated part, which needs no product
            if 0 <= k < L:
                v = q[int(cu_q[b]) + t_last, h % H, geo.dp:geo.dp + geo.rot_dim].float()
                c[k, geo.rw:geo.rw + geo.rot_dim] = v * (8.0 / (scale * float(v @ v)))
        c = c.to(dt)
        nb = -(-L // 16)
        bt[b, :nb] = perm[at:at + nb]
        at += nb
        k = torch.arange(L)
        cache.view(-1, geo.cw)[bt[b, k // 16].long() * 16 + k % 16] = c.float()
        rw = lambda w: torch.einsum("kr,hdr->khd", c[:, :geo.rw].double(), w.double().view(H, -1, geo.rw)).to(dt).double()   # noqa: E731
        rot = torch.zeros(L, geo.rp, dtype=torch.float64)
        rot[:, :geo.rot_dim] = c[:, geo.rw:geo.rw + geo.rot_dim].double()
        keys = torch.cat([rw(wuk), rot[:, None].expand(L, H, geo.rp)], -1)
        s = slice(int(cu_q[b]), int(cu_q[b + 1]))
        rows.append(plain_attention(q[s].double(), keys, rw(wuv), new[b], window, scale, sink.double(), gate[s].double()))
    lat, rot = torch.zeros(S, geo.rw, dtype=dt, device=dev), torch.zeros(S, geo.rp, dtype=dt, device=dev)
    cu_q, cu_k, k_lo = cu_q.to(dev), cu_k.to(dev), torch.tensor(lo, dtype=torch.int32).to(dev)
    ops.latent_gather(cache.to(dt).to(dev), geo, bt.to(dev), 0, cu_k, k_lo, S, lat, rot)
    k, v = ops.gemm(lat, wuk.to(dev)), ops.gemm(lat, wuv.to(dev))
    out = torch.zeros(T, H * geo.vp, dtype=dt, device=dev)
    assert ops.flash_latent_supported(geo)
    ops.flash_latent_prefill(q.to(dev).view(T, -1), k, rot, v, geo, cu_q, cu_k, sink.to(dev), gate.to(dev), out, scale=scale, window=window,
                             max_q=300, rows=T)
    close(out[lead:].view(-1, H, geo.vp), torch.cat(rows), dt)
    assert out[:lead].abs().max() == 0

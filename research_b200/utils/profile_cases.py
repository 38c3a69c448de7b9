"""Small, fixed workloads for Nsight Compute captures: ``python -m research_b200.utils.profile_cases <case>``.

Each case holds well under a few GB on the device, uses inputs larger than the 126 MB L2 where
DRAM figures matter, and launches the kernel of interest a handful of times so a
``--set full`` capture of 1-3 launches ends by itself in a minute or two.
"""

from __future__ import annotations

import sys

import torch

from .. import ops


def case_decode_attn() -> None:
    """paged_decode at the flagship decode shape: 256 sequences x 832 tokens, 14q/2kv heads, D=64."""
    from .microbench import bench_decode_attention

    print(bench_decode_attention(256, 832, 14, 2, 64, 6453.4, iters=3))


def case_decode_attn_d128() -> None:
    from .microbench import bench_decode_attention

    print(bench_decode_attention(64, 2304, 32, 8, 128, 6453.4, iters=3))


def case_gemm_down() -> None:
    """Decode-time down projection of the 0.5B shape: M=256, N=896, K=4864."""
    from .microbench import bench_gemm

    print(bench_gemm(256, 896, 4864, 1688.4, iters=3))


def case_gemm_gateup_8b() -> None:
    """Decode-time gate|up projection of the 8B shape: M=256, N=28672, K=4096 (weights 235 MB, streamed from HBM)."""
    from .microbench import bench_gemm

    print(bench_gemm(256, 28672, 4096, 1688.4, iters=3, bn=256))


def case_gemm_down_8b_cluster() -> None:
    """Decode-time down projection of the 8B shape with split-K over a thread-block cluster: M=256, N=4096, K=14336
    (weights 117 MB per launch, four copies rotated so that every launch streams them from HBM)."""
    import itertools

    ws = [torch.randn(4096, 14336, device="cuda").bfloat16() * 0.05 for _ in range(4)]
    a = torch.randn(256, 14336, device="cuda").bfloat16()
    x = torch.zeros(256, 4096, device="cuda").bfloat16()
    it = itertools.cycle(range(4))
    for _ in range(6):
        ops.gemm(a, ws[next(it)], residual=x, out=x)       # the chooser takes bn 256, 4 slices
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_gemm_qkv_folded_norm() -> None:
    """qkv projection of the 0.5B shape with the RMSNorm folded in: M=256, N=1152, K=896."""
    a = torch.randn(256, 896, device="cuda").bfloat16()
    w = torch.randn(1152, 896, device="cuda").bfloat16() * 0.05
    b = torch.zeros(1152, device="cuda").bfloat16()
    for _ in range(6):
        ops.gemm(a, w, bias=b, norm_eps=1e-6)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_gemm_large() -> None:
    from .microbench import bench_gemm

    print(bench_gemm(4096, 14336, 4096, 1688.4, iters=3))


def case_flash_fwd() -> None:
    """tcgen05 flash attention forward: 8 x 2048 tokens, 32q/8kv heads, D=128, causal."""
    from .microbench import bench_flash_forward

    print(bench_flash_forward(8, 2048, 32, 8, 128, 1688.4, iters=3))


def case_flash_fwd_short() -> None:
    """Flash attention forward at training-rollout lengths: 32 x 512 tokens, 14q/2kv heads, D=64, causal."""
    from .microbench import bench_flash_forward

    print(bench_flash_forward(32, 512, 14, 2, 64, 1688.4, iters=3))


def case_flash_bwd() -> None:
    """tcgen05 flash attention backward: 8 x 2048 tokens, 32q/8kv heads, D=128, causal."""
    from .microbench import bench_flash_backward

    print(bench_flash_backward(8, 2048, 32, 8, 128, 1688.4, iters=3))


def case_decode_step() -> None:
    """Two eager decode steps at batch 256 (for a per-launch time list); the model preset comes from
    RB_PROFILE_MODEL (default: the 0.5B flagship shape), optionally cut to RB_PROFILE_LAYERS layers."""
    from ..inference import EngineConfig, InferenceEngine, SamplingParams
    from ..models import get_preset, init_random_weights

    import os

    over = {"num_layers": int(os.environ["RB_PROFILE_LAYERS"])} if os.environ.get("RB_PROFILE_LAYERS") else {}
    cfg = get_preset(os.environ.get("RB_PROFILE_MODEL", "qwen2.5-0.5b"), **over)   # fewer layers keep big models small
    dev = torch.device("cuda:0")
    w = init_random_weights(cfg, seed=0, dtype=torch.bfloat16, device=dev)
    eng = InferenceEngine(EngineConfig(max_batch_size=256, max_model_len=2048, num_kv_blocks=20000, ignore_eos=True,
                                       use_cuda_graphs=False, max_tokens_per_batch=16384), cfg, w, device=dev)
    g = torch.Generator().manual_seed(0)
    for i in range(256):
        n = int(torch.randint(600, 1000, (1,), generator=g))
        eng.add_request(torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist(), SamplingParams(1.0, 64, seed=i))
    while eng.last_step_rows != (0, 256):
        eng.step()
    torch.cuda.synchronize()
    ops.set_pdl(False)
    # with `ncu --profile-from-start off` only the launches between start() and stop() are captured
    torch.cuda.profiler.start()
    for _ in range(2):
        eng.step()
    torch.cuda.synchronize()
    torch.cuda.profiler.stop()
    print("ok")


def case_gemm_pair() -> None:
    """Two-CTA (``cta_group::2``) GEMM at a training shape: the o projection forward, 4096 x 4096 x 4096, and the gate|up
    projection forward, 4096 x 28672 x 4096 (weights 235 MB: streamed from HBM)."""
    from ..ops.gemm import gemm2

    a = torch.randn(4096, 4096, device="cuda").bfloat16()
    wo = torch.randn(4096, 4096, device="cuda").bfloat16() * 0.05
    wgu = torch.randn(28672, 4096, device="cuda").bfloat16() * 0.05
    out_o = torch.empty(4096, 4096, device="cuda", dtype=torch.bfloat16)
    out_gu = torch.empty(4096, 28672, device="cuda", dtype=torch.bfloat16)
    for _ in range(3):
        gemm2(a, wo, out=out_o)
        gemm2(a, wgu, out=out_gu)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def _optimizer_case(n_params: int):
    """One rank's sharded-optimizer state over ``n_params`` parameters in three chunks (this GPU is its only peer)."""
    from ..parallel.fsdp import FlatBuckets, ShardedAdamW
    from ..parallel.symm import LocalComm

    dev = torch.device("cuda", torch.cuda.current_device())
    comm = LocalComm(dev)
    rows = n_params // 3 // 4096
    shapes = [(f"w{i}", (rows, 4096)) for i in range(3)]
    fb = FlatBuckets(comm, shapes, lambda n: int(n[1:]))
    fb.params.normal_(0, 0.02)
    fb.grads.normal_(0, 0.01)
    return fb, ShardedAdamW(fb, lr=1e-5, max_grad_norm=1.0)


def case_rs_reduce() -> None:
    """Gradient reduce kernel on one GPU: 96 Mi bf16 gradients (192 MB, larger than L2) in three chunks; with one rank
    the launch reads the bucket once and produces the sum of squares (the norm pass of a single-GPU step)."""
    fb, opt = _optimizer_case(96 * 1024 * 1024)
    for _ in range(3):
        for c in range(3):
            opt.reduce_chunk(c)
        opt._reduced.clear()
        opt._passes.clear()
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_adamw_allgather() -> None:
    """Sharded AdamW + parameter write-back on one GPU: 96 Mi parameters (fp32 master and both moments 1.1 GB, bf16
    gradients and parameters 192 MB each), three steps of three chunk launches."""
    fb, opt = _optimizer_case(96 * 1024 * 1024)
    for _ in range(3):
        opt.step()
        fb.grads.normal_(0, 0.01)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_moe_train() -> None:
    """Grouped expert MLP of training, forward + backward, at the Qwen3-30B-A3B layer shape: 4096 tokens, top-8 of 128
    experts, d = 2048, F = 768 (two warm-up passes, then one pass for the launch list)."""
    from ..ops.moe_train import GroupedExperts, GroupedPlan

    class Sink:
        def accumulate_into(self, view):
            return False

    T, k, E, d, F = 4096, 8, 128, 2048, 768
    g = torch.Generator(device="cuda").manual_seed(0)
    h = (torch.randn(T, d, device="cuda", generator=g) * 0.5).bfloat16().requires_grad_(True)
    wgu = (torch.randn(E * 2 * F, d, device="cuda", generator=g) * 0.02).bfloat16()
    wd = (torch.randn(E * d, F, device="cuda", generator=g) * 0.02).bfloat16()
    ggu, gd = torch.empty_like(wgu), torch.empty_like(wd)
    wt, idx = torch.randn(T, E, device="cuda", generator=g).softmax(-1).topk(k, dim=-1)
    wt = wt.contiguous().requires_grad_(True)
    idx32 = idx.to(torch.int32).contiguous()
    dout = (torch.randn(T, d, device="cuda", generator=g) * 0.1).bfloat16()
    for _ in range(3):
        plan = GroupedPlan(idx32, E, d, F)
        GroupedExperts.apply(h, wt, wgu, ggu, wd, gd, plan, Sink()).backward(dout)
        h.grad = wt.grad = None
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_latent_decode() -> None:
    """Latent attention on the cached rows: 256 sequences x 2048 keys, 32 heads, 512 latent + 64 rotated channels (600 MB)."""
    from ..ops.latent import LatentGeometry

    geo, B, L = LatentGeometry(32, 128, 64, 32, 128, 512, 1536), 256, 2048
    cache = torch.randn(B * L // 16, 16, geo.cw, device="cuda").bfloat16()
    bt = torch.randperm(B * L // 16, device="cuda").int().view(B, L // 16).contiguous()
    lens = torch.full((B,), L, dtype=torch.int32, device="cuda")
    qa, out = torch.randn(32, B, geo.cw, device="cuda").bfloat16(), torch.zeros(32, B, geo.rw, dtype=torch.bfloat16, device="cuda")
    sink, gate = torch.zeros(32, device="cuda"), torch.rand(B, 32, device="cuda")
    plan = torch.zeros(ops.latent_units(B, 32, 1) + 1, dtype=torch.int32, device="cuda")
    ops.latent_plan(None, lens, geo, 1, 4096, plan)
    ws = ops.latent_workspace([geo], "cuda")
    for _ in range(3):
        ops.latent_attention(qa, cache, geo, bt, None, lens, sink, gate, out, scale=0.07, window=4096, rows=B, max_q=1, plan=plan, workspace=ws)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_latent_prefill() -> None:
    """Latent attention on multiplied-out keys and values: one prompt of 4096 tokens, 32 heads of 128 + 64 / 128 channels."""
    from ..ops.latent import LatentGeometry

    geo, T = LatentGeometry(32, 128, 64, 32, 128, 512, 1536), 4096
    q, k, v = (torch.randn(T, 32 * n, device="cuda").bfloat16() for n in (192, 128, 128))
    rot, out = torch.randn(T, 64, device="cuda").bfloat16(), torch.empty(T, 32 * 128, dtype=torch.bfloat16, device="cuda")
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    sink, gate = torch.zeros(32, device="cuda"), torch.rand(T, 32, device="cuda")
    for _ in range(3):
        ops.flash_latent_prefill(q, k, rot, v, geo, cu, cu, sink, gate, out, scale=0.07, window=4096, max_q=T, rows=T)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def _recurrent(T: int, seqs: int, gated: bool):
    from ..ops.recurrent import RecurrentGeometry, RecurrentState

    geo = RecurrentGeometry(16, 128, 128, silu=not gated, gated=gated)
    proj = torch.randn(T, geo.proj, device="cuda").bfloat16()
    small, bias, decay = torch.randn(T, 32, device="cuda"), torch.ones(16, device="cuda"), torch.full((16,), 0.97, device="cuda")
    return (proj, small, geo, decay, bias, bias, 15.0, RecurrentState.zeros(geo, seqs, "cuda"), torch.arange(seqs, dtype=torch.int32, device="cuda"))


def case_recurrent_decode() -> None:
    """Matrix memory, one token for each of 256 sequences: 16 heads of 128 x 128 (268 MB of state)."""
    a, out = _recurrent(256, 256, True), torch.empty(256, 2048, device="cuda")
    lens = torch.full((256,), 100, dtype=torch.int32, device="cuda")
    for _ in range(3):
        ops.recurrent_scan(*a, None, lens, out, 256, 256)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_recurrent_prefill() -> None:
    """Matrix memory in chunks: one portion of 4096 tokens, 16 heads of 128 x 128."""
    from ..ops.recurrent import ChunkTable, chunk_workspace

    T = 4096
    a, out = _recurrent(T, 1, True), torch.empty(T, 2048, device="cuda")
    cu, lens = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.tensor([T], dtype=torch.int32, device="cuda")
    table = ChunkTable.make([0, T], 0, "cuda")
    room = torch.empty(chunk_workspace(table.chunks.shape[0], a[2]), dtype=torch.uint8, device="cuda")
    for _ in range(3):
        ops.recurrent_chunks(*a, cu, lens, out, table, room)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_keyvalue_decode() -> None:
    """Keys-as-values attention: 256 sequences x 2048 keys, 16 query heads on 4 kv heads of 128 channels (537 MB of cache)."""
    from ..ops.keyvalue import KeyValueGeometry

    geo, B, L = KeyValueGeometry(16, 4, 128), 256, 2048
    proj = torch.randn(B, geo.proj, device="cuda").bfloat16()
    cache = torch.randn(B * L // 16, 4, 16, 128, device="cuda").bfloat16()
    bt = torch.randperm(B * L // 16, device="cuda").int().view(B, -1)
    lens, sink = torch.full((B,), L, dtype=torch.int32, device="cuda"), torch.zeros(16, device="cuda")
    out = torch.empty(B, 2048, dtype=torch.bfloat16, device="cuda")
    for _ in range(3):
        ops.kv_attention(proj, geo, cache, bt, None, lens, sink, out, scale=0.09, rows=B, max_q=1, n_single=B)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def _time_mix(T: int, seqs: int):
    """32 heads of 64 channels: activations of T rows, state of ``seqs`` sequences."""
    from ..ops.recurrent import RecurrentGeometry, RecurrentState, TimeMix

    geo = RecurrentGeometry(32, 64, 64, silu=False, gated=False)
    proj, norm = torch.randn(T, geo.proj, device="cuda").bfloat16(), torch.ones(2048, device="cuda")
    mix = TimeMix(torch.randn(T, 2048, device="cuda") - 3, torch.zeros(2048, device="cuda"), torch.randn(2048, device="cuda"))
    return proj, geo, mix, RecurrentState.zeros(geo, seqs, "cuda"), torch.arange(seqs, dtype=torch.int32, device="cuda"), norm


def case_time_mix_decode() -> None:
    """Time mixing, one token for each of 256 sequences: 32 heads of 64 x 64 (134 MB of state)."""
    proj, geo, mix, state, slots, norm = _time_mix(256, 256)
    lens, out = torch.full((256,), 100, dtype=torch.int32, device="cuda"), torch.empty(256, 2048, dtype=torch.bfloat16, device="cuda")
    for _ in range(3):
        ops.time_mix_decode(proj, geo, mix, state, slots, lens, norm, 1e-6, out, 256)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_time_mix_prefill() -> None:
    """Time mixing in chunks: one portion of 4096 tokens, 32 heads of 64 x 64."""
    from ..ops.recurrent import ChunkTable, time_mix_workspace

    T = 4096
    proj, geo, mix, state, slots, norm = _time_mix(T, 1)
    cu, lens = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.tensor([T], dtype=torch.int32, device="cuda")
    table, out = ChunkTable.make([0, T], 0, "cuda"), torch.empty(T, 2048, dtype=torch.bfloat16, device="cuda")
    room = torch.empty(time_mix_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device="cuda")
    z = mix.z.clone()
    for _ in range(3):
        mix.z.copy_(z)
        ops.time_mix_chunks(proj, geo, mix, state, slots, cu, lens, norm, 1e-6, out, table, room)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_forget_mix_prefill() -> None:
    """Forget mixing in chunks: one portion of 4096 tokens, 32 heads of 64 x 64."""
    from ..ops.recurrent import ChunkTable, ForgetMix, RecurrentGeometry, RecurrentState, time_mix_workspace

    T, n = 4096, 2048
    geo = RecurrentGeometry(32, 64, 64, silu=True, gated=False, form="forget")
    proj, z = torch.randn(T, geo.proj, device="cuda").bfloat16(), torch.randn(T, n, device="cuda") + 3
    mix = ForgetMix(z.clone(), torch.zeros(n, device="cuda"), torch.rand(n, device="cuda") * 0.5, torch.empty(T, 2 * n, dtype=torch.bfloat16, device="cuda"))
    state, slots = RecurrentState.zeros(geo, 1, "cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    cu, lens = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.tensor([T], dtype=torch.int32, device="cuda")
    table, out, norm = ChunkTable.make([0, T], 0, "cuda"), torch.empty(T, n, dtype=torch.bfloat16, device="cuda"), torch.ones(n, device="cuda")
    room = torch.empty(time_mix_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device="cuda")
    for _ in range(3):
        mix.z.copy_(z)
        ops.time_mix_chunks(proj, geo, mix, state, slots, cu, lens, norm, 1e-6, out, table, room)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def _delta(T: int, seqs: int):
    """16 heads of 128 channels: rows, factors and steps of T tokens, state of ``seqs`` sequences."""
    from ..ops.recurrent import DeltaRule, RecurrentGeometry, RecurrentState

    geo = RecurrentGeometry(16, 128, 128, silu=False, gated=False, form="delta", groups=16)
    rows = torch.randn(T, geo.channels, device="cuda").bfloat16()
    rule = DeltaRule(torch.full((T, 32), 128 ** -0.5, device="cuda"), torch.cat([-torch.rand(T, 16, device="cuda") * 0.1, torch.rand(T, 16, device="cuda")], 1))
    return rows, geo, rule, RecurrentState.zeros(geo, seqs, "cuda"), torch.arange(seqs, dtype=torch.int32, device="cuda")


def case_delta_prefill() -> None:
    """Delta rule in chunks: one portion of 4096 tokens, 16 heads of 128 x 128."""
    from ..ops.recurrent import ChunkTable, delta_workspace

    T = 4096
    rows, geo, rule, state, slots = _delta(T, 1)
    cu, lens = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.tensor([T], dtype=torch.int32, device="cuda")
    table, out = ChunkTable.make([0, T], 0, "cuda"), torch.empty(T, 2048, device="cuda")
    room = torch.empty(delta_workspace(table.chunks.shape[0], geo), dtype=torch.uint8, device="cuda")
    for _ in range(3):
        ops.delta_chunks(rows, geo, rule, state, slots, cu, lens, out, table, room)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_delta_decode() -> None:
    """Delta rule, one token for each of 256 sequences: 16 heads of 128 x 128 (268 MB of state)."""
    rows, geo, rule, state, slots = _delta(256, 256)
    lens, out = torch.full((256,), 100, dtype=torch.int32, device="cuda"), torch.empty(256, 2048, device="cuda")
    for _ in range(3):
        ops.recurrent_scan(rows, None, geo, None, None, None, 1.0, state, slots, None, lens, out, 256, 256, mix=rule)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_delta_rows() -> None:
    """Convolutions of 4 taps, SiLU and units of 4096 tokens: 16 heads of 128 channels each of queries, keys and values."""
    T = 4096
    rows, geo, rule, _, slots = _delta(T, 1)
    proj, small = torch.randn(T, geo.proj, device="cuda").bfloat16(), torch.randn(T, 32, device="cuda")
    hist, ones = torch.zeros(2, 3, geo.channels, dtype=torch.bfloat16, device="cuda"), torch.ones(16, device="cuda")
    cu, pos = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.arange(T, dtype=torch.int32, device="cuda")
    for _ in range(3):
        ops.delta_rows(proj, small, geo, torch.ones(4, geo.channels, device="cuda"), hist, cu, pos, slots, ones, ones, rows, rule)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def _grouped(T: int, rows_cached: int, conv: bool):
    from ..ops.grouped import GroupedCache, GroupedGeometry

    geo = GroupedGeometry(16, 4, 128, 128, 4 if conv else 1, conv, "head" if conv else "projection", 64, conv)
    cache = GroupedCache(*(torch.randn(rows_cached // 16, 4, 16, 128, device="cuda").bfloat16() for _ in range(2)),
                         torch.zeros(2, 3, geo.channels, device="cuda").bfloat16() if conv else None)
    return geo, cache, torch.randn(T, geo.proj, device="cuda").bfloat16(), torch.empty(T, 2048, dtype=torch.bfloat16, device="cuda")


def _case_append(conv: bool) -> None:
    T = 4096
    geo, cache, proj, q = _grouped(T, T, conv)
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    cu, slot = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    ones, table = torch.ones(2048, device="cuda"), ops.frequency_table(T, [0.9 ** i for i in range(32)], 1.0, "cuda")
    for _ in range(3):
        ops.grouped_append(proj, geo, conv=torch.ones(4, geo.channels, device="cuda") if conv else None, cache=cache, cu_q=cu, positions=pos, state_slots=slot,
                           slots=pos, q_norm=None if conv else ones, k_norm=None if conv else ones, eps=1e-6, table=table, q=q)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


def case_grouped_append() -> None:
    """Norm over the projection, rotation and cache append of 4096 tokens: 16 query heads on 4 kv heads of 128 channels."""
    _case_append(False)


def case_grouped_append_conv() -> None:
    """The same with convolutions of 4 taps and a norm per head."""
    _case_append(True)


def case_grouped_decode() -> None:
    """Attention over cached keys and values: 256 sequences x 2048 keys, 16 query heads on 4 kv heads of 128 channels (1 GB of cache)."""
    B, L = 256, 2048
    geo, cache, _, q = _grouped(B, B * L, False)
    bt = torch.randperm(B * L // 16, device="cuda").int().view(B, -1)
    lens, out = torch.full((B,), L, dtype=torch.int32, device="cuda"), torch.empty(B, 2048, dtype=torch.bfloat16, device="cuda")
    q.normal_()
    for _ in range(3):
        ops.grouped_attention(q, geo, cache, bt, None, lens, out, scale=0.09, rows=B, max_q=1, n_single=B)
    torch.cuda.synchronize()
    ops.check_status()
    print("ok")


CASES = {k[5:]: v for k, v in globals().items() if k.startswith("case_")}

if __name__ == "__main__":
    name = sys.argv[1] if len(sys.argv) > 1 else "decode_attn"
    CASES[name]()

"""Prefill and decode throughput of a layer-stack model beside the closest Hugging Face style model of equal size.

``bench.py --workload stack`` runs it. For every size two engines are built with random weights: the latent-attention
stack and a Llama-type model with the same width, layers, feed-forward, vocabulary and heads (grouped queries, head size
128). Measured with CUDA events, after warm-up:

* decode: one captured decode step at the given batch and context, replayed;
* prefill: one packed pass over a whole prompt;
* every kernel of a layer on its own at those shapes, L2 flushed before each launch, against its roofline: the larger of
  bytes that must move / measured copy bandwidth and operations / measured tensor throughput.
"""

from __future__ import annotations

import json
import statistics
from dataclasses import dataclass
from pathlib import Path

import torch

from .. import ops
from ..inference import EngineConfig, InferenceEngine
from ..models import LazyRandomWeights
from ..models.config import ModelConfig
from ..models.stack import ClampedGluSpec, LatentAttentionSpec, RotarySpec, uniform_stack
from .timing import flush_l2, time_cuda


@dataclass(frozen=True)
class Size:
    name: str
    width: int
    layers: int
    heads: int
    kv_heads: int
    ff: int
    vocab: int
    q_rank: int
    kv_rank: int = 512
    window: int = 4096


SIZES = (Size("1b", 2048, 8, 16, 4, 8192, 32000, 1024), Size("7b", 4096, 8, 32, 8, 14336, 32000, 1536))


def peaks() -> tuple[float, float, str]:
    """(bytes/s, bf16 flop/s, origin): the measured figures when the file is there."""
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def configs(s: Size):
    mixer = LatentAttentionSpec(s.heads, 128, 64, 128, s.kv_rank, s.q_rank, 192 ** -0.5, s.window, RotarySpec(64, 5e5))
    stack = uniform_stack("Lulezen", vocab=s.vocab, width=s.width, num_layers=s.layers, mixer=mixer, mlp=ClampedGluSpec(s.ff, 7.0),
                          logit_softcap=30.0)
    llama = ModelConfig(family="llama", vocab_size=s.vocab, hidden_size=s.width, num_layers=s.layers, num_heads=s.heads,
                        num_kv_heads=s.kv_heads, head_dim=128, intermediate_size=s.ff, rope_theta=5e5, tie_word_embeddings=False,
                        attention_bias=False)
    return stack, llama


def _engine(cfg, batch: int, context: int, prompt: int) -> InferenceEngine:
    w = LazyRandomWeights(cfg, seed=0, dtype=torch.bfloat16, device="cuda")
    blocks = batch * (-(-context // 16)) + 2 * (-(-prompt // 16))
    return InferenceEngine(EngineConfig(cache_type="none", max_batch_size=batch, max_model_len=max(context, prompt) + 64,
                                        max_tokens_per_batch=prompt, num_kv_blocks=blocks, ignore_eos=True,
                                        graph_batch_sizes=(batch,)), cfg, w, device="cuda")


def _stage_decode(r, batch: int, context: int) -> None:
    """Fill the decode staging: every row one token behind a context of ``context`` keys in blocks of its own."""
    per = -(-context // 16)
    perm = torch.randperm(batch * per, generator=torch.Generator().manual_seed(0)).int().view(batch, per)
    r.bt_host[:batch, :per] = perm
    r.bt_dev[:batch, :per] = perm.to(r.device)
    mb, m = r.max_batch, r.meta_host
    m[0:batch] = 1
    m[mb:mb + batch] = context - 1
    m[2 * mb:2 * mb + batch] = perm[:, (context - 1) // 16] * 16 + (context - 1) % 16
    m[3 * mb:3 * mb + batch] = context
    r.meta_dev.copy_(m)


def time_decode(eng: InferenceEngine, batch: int, context: int, iters: int = 30) -> float:
    """Milliseconds of one captured decode step (the weights and the cache exceed L2)."""
    r = eng.runner
    _stage_decode(r, batch, context)
    g = r.graphs[r.bucket(batch)]
    for _ in range(5):
        g.replay()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        flush_l2()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record()
        g.replay()
        e.record()
        torch.cuda.synchronize()
        times.append(s.elapsed_time(e))
    return statistics.median(times)


def time_prefill(eng: InferenceEngine, prompt: int, iters: int = 8) -> float:
    """Milliseconds of one packed pass over a prompt, sampling included."""
    r, o = eng.runner, eng.runner._pf_offsets()
    ph, n = r.pf_host, prompt
    ph[o["tokens"]:o["tokens"] + n] = torch.arange(n, dtype=torch.int32) % 1000
    ph[o["positions"]:o["positions"] + n] = torch.arange(n, dtype=torch.int32)
    ph[o["slots"]:o["slots"] + n] = torch.arange(n, dtype=torch.int32)
    ph[o["cu_q"]:o["cu_q"] + 2] = torch.tensor([0, n], dtype=torch.int32)
    ph[o["seq_lens"]] = n
    ph[o["sample_rows"]] = n - 1
    r.bt_host[0, :-(-n // 16)] = torch.arange(-(-n // 16), dtype=torch.int32)
    return time_cuda(lambda: r.prefill(1, n, n, -(-n // 16)), iters=iters, flush=False)["median_ms"]


# ------------------------------------------------------------------------------- kernels one by one
class _Table:
    def __init__(self):
        self.bw, self.fl, self.origin = peaks()
        self.rows: dict[str, dict] = {}

    def add(self, name: str, fn, nbytes: float, flops: float) -> None:
        us = time_cuda(fn, iters=15)["median_ms"] * 1e3
        ideal = max(nbytes / self.bw, flops / self.fl) * 1e6
        self.rows[name] = {"us": round(us, 2), "roofline_us": round(ideal, 2), "of_roofline": round(ideal / us, 3)}

    def gemm(self, name: str, M: int, N: int, K: int, call, out_bytes: int = 2, out_cols: int | None = None) -> None:
        self.add(name, call, 2 * (M * K + N * K) + out_bytes * M * (out_cols or N), 2.0 * M * N * K)


def stack_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """Time every kernel of the first layer at ``T`` rows: decode rows with ``context`` keys each, or one prompt of T tokens."""
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    lw = r.layers[0]
    g, b, m = lw.geo, r.bufs[lw.geo], lw.spec.mixer
    H, d = g.heads, cfg.hidden_size
    x, xb, y = r.x[:T], r.xb[:T], r.y[:T]
    pos = torch.full((T,), context - 1, dtype=torch.int32, device="cuda") if decode else torch.arange(T, dtype=torch.int32, device="cuda")
    slots = r.d_slots[:T] if decode else pos
    n_short = T if decode else 0
    t.gemm("joint down projection", T, g.proj, r.wp, lambda: ops.gemm(xb, lw.wproj, out=b.proj[:T], out_f32=True), 4)
    t.add("norms + rotation + append", lambda: ops.latent_append(b.proj[:T], g, lw.q_norm, lw.kv_norm, cfg.norm_eps, pos, slots, lw.table,
                                                                 lw.cache, b.cq, b.gate), T * (4 * g.proj + 2 * g.qp + 2 * g.cw), 0)
    q = b.q[:T]
    t.gemm("query up projection", T, q.shape[1], g.qp, lambda: ops.gemm(b.cq[:T], lw.wuq, out=q))
    rot_bytes = T * H * (2 * 2 * (g.dp + g.rp) if decode else 2 * 2 * g.rp)
    t.add("query rotation", lambda: ops.latent_query(q, g, pos, lw.table, n_short, b.qn, b.qa), rot_bytes, 0)
    if decode:
        bt, lens = r.bt_dev[:T], r.d_lens[:T]
        span = min(context, m.window)
        plan = r.decode_plans[(g, m.window)]
        ops.latent_plan(None, lens, g, 1, m.window, plan)
        t.add("absorb W_uk", lambda: ops.head_gemm_absorb(b.qn, lw.wuk, b.qa, T), 2 * H * (g.dp * g.rw + T * (g.dp + g.rw)), 2.0 * T * H * g.dp * g.rw)
        t.add("attention", lambda: ops.latent_attention(b.qa, lw.cache, g, bt, None, lens, lw.sink, b.gate, b.ol, scale=m.scale, window=m.window,
                                                        rows=T, max_q=1, plan=plan, workspace=r.attn_ws),
              2 * T * (span * g.cw + H * (g.cw + g.rw)), 2.0 * T * H * span * (g.cw + g.rw))
        t.add("expand W_uv", lambda: ops.head_gemm_expand(b.ol, lw.wuv, b.attn, T), 2 * H * (g.vp * g.rw + T * (g.vp + g.rw)), 2.0 * T * H * g.vp * g.rw)
    else:
        bt = torch.arange(-(-T // 16), dtype=torch.int32, device="cuda")[None].contiguous()
        cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
        lo = torch.zeros(1, dtype=torch.int32, device="cuda")
        lat = torch.empty(T, g.rw, dtype=torch.bfloat16, device="cuda")
        rot = torch.empty(T, g.rp, dtype=torch.bfloat16, device="cuda")
        t.add("gather latents", lambda: ops.latent_gather(lw.cache, g, bt, 0, cu, lo, T, lat, rot), 2 * 2 * T * g.cw, 0)
        k, v = ops.gemm(lat, lw.wuk), ops.gemm(lat, lw.wuv)
        t.gemm("keys", T, k.shape[1], g.rw, lambda: ops.gemm(lat, lw.wuk, out=k))
        t.gemm("values", T, v.shape[1], g.rw, lambda: ops.gemm(lat, lw.wuv, out=v))
        pairs = sum(min(i + 1, m.window) for i in range(T))
        t.add("attention", lambda: ops.flash_latent_prefill(q, k, rot, v, g, cu, cu, lw.sink, b.gate, b.attn, scale=m.scale, window=m.window,
                                                            max_q=T, rows=T),
              2 * T * H * (2 * g.dp + g.rp + 2 * g.vp), 2.0 * pairs * H * (g.dp + g.rp + g.vp))
    t.gemm("output projection", T, r.wp, H * g.vp, lambda: ops.gemm(b.attn[:T], lw.wo, out=y, out_f32=True), 4)
    t.add("norm + residual", lambda: ops.layernorm_residual(y, lw.norm1[0], lw.norm1[1], cfg.norm_eps, x, xb), T * d * 14, 0)
    act = r._act[:T * lw.ffp].view(T, lw.ffp)
    t.gemm("gate|up + unit", T, 2 * lw.ffp, r.wp, lambda: ops.gemm(xb, lw.wgu, out=act, bn=r.glu_bn, swiglu=True, glu_limit=lw.glu.limit), 2, lw.ffp)
    t.gemm("down projection", T, r.wp, lw.ffp, lambda: ops.gemm(act, lw.wd, out=y, out_f32=True), 4)
    if decode:
        lg = r.logits_padded[:T]
        t.gemm("head + cap", T, r.vp, r.wp, lambda: r._head(r.hl[:T], lg), 4)
    return t.rows


def llama_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    lw = r.layers[0]
    d, Hq, Hkv, D = cfg.hidden_size, r.Hq, r.Hkv, r.D
    eps = cfg.rms_norm_eps
    x = torch.randn(T, d, device="cuda").bfloat16()
    h = torch.empty_like(x)
    pos = torch.full((T,), context - 1, dtype=torch.int32, device="cuda") if decode else torch.arange(T, dtype=torch.int32, device="cuda")
    slots = r.d_slots[:T] if decode else pos
    fold = eps if r.fold_norm else None
    qkv = torch.empty(T, lw.wqkv.shape[0], dtype=torch.bfloat16, device="cuda")
    t.gemm("qkv projection", T, qkv.shape[1], d, lambda: ops.gemm(x, lw.wqkv, out=qkv, norm_eps=fold))
    q = torch.empty(T, Hq * D, dtype=torch.bfloat16, device="cuda")
    t.add("rotation + append", lambda: ops.rope_kv_append(qkv, pos, slots, r.rope, r.k_cache[0], r.v_cache[0], Hq, Hkv, D, q_out=q),
          2 * 2 * T * qkv.shape[1], 0)
    q3, o = q.view(T, Hq, D), torch.empty(T, Hq, D, dtype=torch.bfloat16, device="cuda")
    if decode:
        splits = ops.decode_num_splits(T, Hkv, r.max_model_len, head_dim=D) if T <= 64 else 1
        t.add("attention", lambda: ops.paged_decode(q3, r.k_cache[0], r.v_cache[0], r.bt_dev[:T], r.d_lens[:T], r.scale, splits, out=o,
                                                    workspace=r.dec_ws), 2 * T * (2 * context * Hkv * D + 2 * Hq * D), 4.0 * T * Hq * context * D)
    else:
        bt = torch.arange(-(-T // 16), dtype=torch.int32, device="cuda")[None].contiguous()
        cu, sl = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.tensor([T], dtype=torch.int32, device="cuda")
        t.add("attention", lambda: ops.paged_prefill(q3, r.k_cache[0], r.v_cache[0], bt, cu, sl, T, r.scale, 0, out=o),
              2 * T * D * (2 * Hq + 2 * Hkv), 4.0 * (T * (T + 1) / 2) * Hq * D)
    t.gemm("output projection", T, d, Hq * D, lambda: ops.gemm(o.view(T, Hq * D), lw.wo, residual=x, out=x))
    t.add("norm", lambda: ops.rmsnorm(x, lw.ln2, eps, out=h), 4 * T * d, 0)
    act = torch.empty(T, r.F, dtype=torch.bfloat16, device="cuda")
    t.gemm("gate|up + unit", T, 2 * r.F, d, lambda: ops.gemm(h, lw.wgu, out=act, bn=r.swiglu_bn, swiglu=True, norm_eps=fold), 2, r.F)
    t.gemm("down projection", T, d, r.F, lambda: ops.gemm(act, lw.wd, residual=x, out=x))
    if decode:
        t.gemm("head", T, cfg.vocab_size, d, lambda: ops.gemm(h, r.lm_head, out=r.a_logits[:T], out_f32=True), 4)
    return t.rows


def run(sizes: tuple[str, ...] = (), batches: tuple[int, ...] = (1, 64, 256), context: int = 2048, prompts: tuple[int, ...] = (512, 4096),
        kernels: bool = True) -> dict:
    out: dict = {"peaks": dict(zip(("hbm_bytes_s", "bf16_flop_s", "origin"), peaks())), "context": context, "sizes": {}}
    for s in SIZES:
        if sizes and s.name not in sizes:
            continue
        res: dict = {"shape": {k: getattr(s, k) for k in ("width", "layers", "heads", "kv_heads", "ff", "vocab", "q_rank", "kv_rank", "window")}}
        for label, cfg in zip(("lulezen", "llama"), configs(s)):
            one: dict = {"params_m": round(cfg.num_params() / 1e6), "decode": {}, "prefill": {}, "decode_kernels": {}, "prefill_kernels": {}}
            table = stack_kernels if label == "lulezen" else llama_kernels
            for B in batches:
                eng = _engine(cfg, max(B, 2), context, max(prompts))
                ms = time_decode(eng, B, context)
                one["decode"][B] = {"ms": round(ms, 4), "tok_s": round(B / ms * 1e3)}
                if B == batches[-1]:
                    if kernels:
                        one["decode_kernels"] = table(eng, B, context, True)
                    for n in prompts:
                        ms = time_prefill(eng, n)
                        one["prefill"][n] = {"ms": round(ms, 3), "tok_s": round(n / ms * 1e3)}
                    if kernels:
                        one["prefill_kernels"] = table(eng, prompts[-1], context, False)
                ops.check_status()
                eng.shutdown()
                del eng
                torch.cuda.empty_cache()
            res[label] = one
        out["sizes"][s.name] = res
    return out

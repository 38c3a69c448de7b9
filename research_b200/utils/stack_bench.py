"""Prefill and decode throughput of layer-stack models beside the closest Hugging Face style model of equal size.

``bench.py --workload stack`` runs it (``--designs``, ``--sizes`` choose). For every size two engines are built with random
weights: Lulezen (latent attention) beside a Llama-type model, Zamusun (recurrent mixers, keys-as-values attention, routed
experts, a looped pair of layers) and Fogurax (grouped attention with convolutions or chunks, attention beside time mixing, routed and
shared experts, a per-layer token input) beside a Qwen3-MoE-type model, Sumitar (gated delta rule, attention beside forget mixing, identity
experts, normed powers) beside Fogurax, each with the same width, layer runs, feed-forward,
vocabulary and heads (grouped queries, head size 128). Measured with CUDA events, after warm-up:

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
from ..models.stack import (DESIGNS as STACK_DESIGNS, BandScaling, ClampedGluSpec, DeltaRuleSpec, ExpertsRouting, ExpertsSpec, ForgetMixSpec, GluSpec,
                            GroupedAttentionSpec, KeyValueAttentionSpec, LatentAttentionSpec, LayerSpec, LayerStackConfig, LightningSpec, LoopSpec,
                            MatrixMemorySpec, NormedPairSpec, ParallelSpec, PolyNormSpec, QueryTemperature, RotarySpec, TimeMixSpec, TokenSideSpec,
                            YarnScaling, uniform_stack)
from ..inference.stack_parts import DensePart
from ..ops import experts as ex
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


@dataclass(frozen=True)
class ExpertSize:
    name: str
    width: int
    runs: int                # layer runs; two of the layers are looped twice, so there are runs - 2 layers
    heads: int
    kv_heads: int
    experts: int
    top: int
    ff: int
    vocab: int


EXPERT_SIZES = (ExpertSize("w2048", 2048, 8, 16, 4, 64, 8, 768, 32000), ExpertSize("w4096", 4096, 8, 32, 8, 16, 2, 4096, 32000))


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


def expert_configs(s: ExpertSize):
    H = s.heads
    memory, linear = MatrixMemorySpec(H, 128, 128, 15.0), LightningSpec(H, 128, 128, tuple(1 - 2.0 ** -(2 + 6 * h / H) for h in range(H)))
    attention = KeyValueAttentionSpec(H, s.kv_heads, 128, 128 ** -0.5, QueryTemperature(0.1, 1024))
    mlp = ExpertsSpec(s.experts, s.top, ClampedGluSpec(s.ff, 7.0))
    kinds = (memory, linear, attention)
    stack = LayerStackConfig("Zamusun", s.vocab, s.width, tuple(LayerSpec(kinds[i % 3], mlp) for i in range(s.runs - 2)), loop=LoopSpec(0, 2, 2))
    moe = ModelConfig(family="qwen3_moe", vocab_size=s.vocab, hidden_size=s.width, num_layers=s.runs, num_heads=H, num_kv_heads=s.kv_heads,
                      head_dim=128, intermediate_size=s.ff, rope_theta=5e5, tie_word_embeddings=True, attention_bias=False, qk_norm=True,
                      num_experts=s.experts, num_experts_per_tok=s.top, moe_intermediate_size=s.ff)
    return stack, moe


def fogurax_stack(s: ExpertSize, layers: int, conv: int = 4, reach: int = 4096, side: int = 256) -> LayerStackConfig:
    """Every third layer has attention in chunks, convolutions on the projections, or attention beside time mixing; heads of 128
    channels in attention and 64 in time mixing."""
    H, G, kinds = s.heads, s.kv_heads, STACK_DESIGNS["Fogurax"].mixers

    def rot(interleaved, scaling=None):
        return RotarySpec(64, 5e5, interleaved, scaling)

    def heads(form, r, taps=1, size=0):
        return GroupedAttentionSpec(form, H, G, 128, 128, 128 ** -0.5, r, taps, size)

    chunked = heads(kinds["attention_2"], rot(False, YarnScaling(4.0, 4096, 32.0, 1.0)), size=reach)
    conved = heads(kinds["attention"], rot(True, BandScaling(8.0, 1.0, 4.0, 8192)), conv)
    both = ParallelSpec("parallel", heads(kinds["parallel"].left, rot(True), size=reach), TimeMixSpec(2 * H, 64, 64), 1.0, 1.0)
    mlp = ExpertsSpec(s.experts, s.top, GluSpec(s.ff), ExpertsRouting("sigmoid", False, True), GluSpec(s.ff))
    return LayerStackConfig("Fogurax", s.vocab, s.width, tuple(LayerSpec((chunked, conved, both)[i % 3], mlp) for i in range(layers)),
                            residual_mult=0.5, token_side=TokenSideSpec(side))


def fogurax_configs(s: ExpertSize):
    return fogurax_stack(s, s.runs), expert_configs(s)[1]


def sumitar_stack(s: ExpertSize, layers: int, conv: int = 4, reach: int = 4096) -> LayerStackConfig:
    """Two layers of the delta rule (heads of 128 channels), then attention beside forget mixing (heads of 64); the first feed-forward has normed
    powers, the others route, one choice in sixteen an identity."""
    H, kinds = s.heads, STACK_DESIGNS["Sumitar"].mixers
    rule = DeltaRuleSpec(H, H, 128, 128, conv)
    left = GroupedAttentionSpec(kinds["parallel"].left, H, s.kv_heads, 128, 128, 128 ** -0.5, RotarySpec(64, 5e5), 1, reach)
    both = NormedPairSpec("parallel", left, ForgetMixSpec(2 * H, 64, 64))
    plain = s.experts // 16
    mlp = ExpertsSpec(s.experts - plain, s.top, GluSpec(s.ff), ExpertsRouting(normalize=False, correction=True, shared_gate=True), GluSpec(s.ff), plain)
    return LayerStackConfig("Sumitar", s.vocab, s.width, tuple(LayerSpec(both if i % 3 == 2 else rule, PolyNormSpec(s.top * s.ff) if i == 0 else mlp)
                                                               for i in range(layers)))


def sumitar_configs(s: ExpertSize):
    return sumitar_stack(s, s.runs), fogurax_stack(s, s.runs)


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
    m[7 * mb:7 * mb + batch] = torch.arange(batch, dtype=torch.int32)
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
    ph[o["state_slots"]] = 0
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


def latent_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """Time every kernel of the first layer at ``T`` rows: decode rows with ``context`` keys each, or one prompt of T tokens."""
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    layer = r.layers[0]
    lw, part, cache = layer.mix, layer.mixer, r.runs[0].cache
    g, b, m = lw.geo, part.bufs[lw.geo], lw.spec
    H, d = g.heads, cfg.hidden_size
    x, xb, y = r.x[:T], r.xb[:T], r.y[:T]
    pos = torch.full((T,), context - 1, dtype=torch.int32, device="cuda") if decode else torch.arange(T, dtype=torch.int32, device="cuda")
    slots = r.d_slots[:T] if decode else pos
    n_short = T if decode else 0
    t.gemm("joint down projection", T, g.proj, r.wp, lambda: ops.gemm(xb, lw.wproj, out=b.proj[:T], out_f32=True), 4)
    t.add("norms + rotation + append", lambda: ops.latent_append(b.proj[:T], g, lw.q_norm, lw.kv_norm, cfg.norm_eps, pos, slots, lw.table,
                                                                 cache, b.cq, b.gate), T * (4 * g.proj + 2 * g.qp + 2 * g.cw), 0)
    q = b.q[:T]
    t.gemm("query up projection", T, q.shape[1], g.qp, lambda: ops.gemm(b.cq[:T], lw.wuq, out=q))
    rot_bytes = T * H * (2 * 2 * (g.dp + g.rp) if decode else 2 * 2 * g.rp)
    t.add("query rotation", lambda: ops.latent_query(q, g, pos, lw.table, n_short, b.qn, b.qa), rot_bytes, 0)
    if decode:
        bt, lens = r.bt_dev[:T], r.d_lens[:T]
        span = min(context, m.window)
        plan = part.decode_plans[(g, m.window)]
        ops.latent_plan(None, lens, g, 1, m.window, plan)
        t.add("absorb W_uk", lambda: ops.head_gemm_absorb(b.qn, lw.wuk, b.qa, T), 2 * H * (g.dp * g.rw + T * (g.dp + g.rw)), 2.0 * T * H * g.dp * g.rw)
        t.add("attention", lambda: ops.latent_attention(b.qa, cache, g, bt, None, lens, lw.sink, b.gate, b.ol, scale=m.scale, window=m.window,
                                                        rows=T, max_q=1, plan=plan, workspace=part.workspace),
              2 * T * (span * g.cw + H * (g.cw + g.rw)), 2.0 * T * H * span * (g.cw + g.rw))
        t.add("expand W_uv", lambda: ops.head_gemm_expand(b.ol, lw.wuv, b.attn, T), 2 * H * (g.vp * g.rw + T * (g.vp + g.rw)), 2.0 * T * H * g.vp * g.rw)
    else:
        bt = torch.arange(-(-T // 16), dtype=torch.int32, device="cuda")[None].contiguous()
        cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
        lo = torch.zeros(1, dtype=torch.int32, device="cuda")
        lat = torch.empty(T, g.rw, dtype=torch.bfloat16, device="cuda")
        rot = torch.empty(T, g.rp, dtype=torch.bfloat16, device="cuda")
        t.add("gather latents", lambda: ops.latent_gather(cache, g, bt, 0, cu, lo, T, lat, rot), 2 * 2 * T * g.cw, 0)
        k, v = ops.gemm(lat, lw.wuk), ops.gemm(lat, lw.wuv)
        t.gemm("keys", T, k.shape[1], g.rw, lambda: ops.gemm(lat, lw.wuk, out=k))
        t.gemm("values", T, v.shape[1], g.rw, lambda: ops.gemm(lat, lw.wuv, out=v))
        pairs = sum(min(i + 1, m.window) for i in range(T))
        t.add("attention", lambda: ops.flash_latent_prefill(q, k, rot, v, g, cu, cu, lw.sink, b.gate, b.attn, scale=m.scale, window=m.window,
                                                            max_q=T, rows=T),
              2 * T * H * (2 * g.dp + g.rp + 2 * g.vp), 2.0 * pairs * H * (g.dp + g.rp + g.vp))
    t.gemm("output projection", T, r.wp, H * g.vp, lambda: ops.gemm(b.attn[:T], lw.wo, out=y, out_f32=True), 4)
    t.add("norm + residual", lambda: ops.layernorm_residual(y, layer.norm1[0], layer.norm1[1], cfg.norm_eps, x, xb, d), T * d * 14, 0)
    ff = layer.ff
    act = layer.feed_forward.act[:T * ff.ffp].view(T, ff.ffp)
    t.gemm("gate|up + unit", T, 2 * ff.ffp, r.wp, lambda: ops.gemm(xb, ff.wgu, out=act, bn=256, swiglu=True, glu_limit=ff.spec.limit), 2, ff.ffp)
    t.gemm("down projection", T, r.wp, ff.ffp, lambda: ops.gemm(act, ff.wd, out=y, out_f32=True), 4)
    if decode:
        lg = r.logits_padded[:T]
        t.gemm("head + cap", T, r.vp, r.wp, lambda: r._head(r.hl[:T], lg), 4)
    return t.rows


def _routed(t: _Table, T: int, E: int, k: int, d: int, ff: int, up, down, unit=None, others: dict | None = None) -> None:
    """Rows of the routed experts: ``others`` are the small launches around the two grouped products."""
    n = T * k
    active = min(E, n)
    for name, (fn, nbytes) in (others or {}).items():
        t.add(name, fn, nbytes, 0)
    t.add("experts gate|up", up, 2 * (n * d + active * 2 * ff * d + n * (ff if unit is None else 2 * ff)), 4.0 * n * d * ff)
    if unit is not None:
        t.add("experts unit", unit, 2 * 3 * n * ff, 0)
    t.add("experts down", down, 2 * (n * ff + active * ff * d + n * d), 2.0 * n * d * ff)


def expert_stack_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """The first layer of every kind of mixer, the routed experts and what joins them."""
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    d, eps = cfg.hidden_size, cfg.norm_eps
    x, h, y = r.x[:T], r.xb[:T], r.y[:T]
    h.normal_()
    b = r._decode_batch(T) if decode else _prompt_batch(r, T)
    seen = set()
    for run in r.runs:
        lw = run.layer
        w, part, kind = lw.mix, lw.mixer, lw.spec.mixer.type
        if kind in seen:
            continue
        seen.add(kind)
        g, plan = w.geo, part.plan(b)
        proj = part.proj[:T * g.proj].view(T, g.proj)
        t.gemm(f"{kind}: joint projection", T, w.wproj.shape[0], r.wp, lambda: r._project(lw, h))
        if kind == "attention":
            H, G, D, m = g.heads, g.kv_heads, g.dp, w.spec
            out = part.out[:T * H * D].view(T, H * D)
            t.add("attention: temperature + append", lambda: ops.kv_append(proj, g, b.positions, b.slots, m.q_temp.coef, m.q_temp.every, run.cache),
                  2 * T * D * (2 * H + 2 * G), 0)
            fn = lambda: ops.kv_attention(proj, g, run.cache, b.block_tables, b.cu_q, b.seq_lens, w.sink, out, scale=m.scale, rows=T, max_q=b.max_new,
                                          n_single=b.n_single, workspace=part.workspace, splits=plan.get(g, 1))
            if decode:
                t.add("attention: attention", fn, 2 * T * (context * G * D + 3 * H * D), 4.0 * T * H * context * D)
            else:
                t.add("attention: attention", fn, 2 * T * D * (3 * H + G), 4.0 * (T * (T + 1) / 2) * H * D)
            n = H * D
        else:
            H, n = g.heads, g.heads * g.vp
            o, out = part.o[:T * n].view(T, n), part.out[:T * n].view(T, n)
            small = r._project(lw, h)
            io = T * H * (2 * (2 * g.kp + g.vp) + 4 * g.vp)
            state = 2 * 4 * H * g.kp * (g.vp + (1 if g.gated else 0))
            t.add(f"{kind}: recurrence", lambda: part.recur(w, run.cache, proj, small, o, b, plan), io + state * b.rows,
                  T * H * (4.0 * g.kp * g.vp + (0 if decode else 2.0 * 64 * (g.kp + g.vp))))
            t.add(f"{kind}: norm + gate", lambda: ops.gated_norm(o, w.norm, proj[:, g.offsets[3]:], g, eps, out, g.gated), T * n * 8, 0)
        t.gemm(f"{kind}: output projection", T, r.wp, n, lambda: ops.gemm(out, w.wo, bias=getattr(w, "bo", None), out=y, out_f32=True), 4)
    lw = r.layers[0]
    logits = r._project(lw, h)[:, lw.mix_small:]
    w, g = lw.ff, lw.ff.geo
    sc = lw.feed_forward.scratch[g]
    _routed(t, T, g.experts, g.top, d, g.ff, lambda: ex.experts_up(g, sc, w.wgu, T), lambda: ex.experts_down(g, sc, w.wd), None,
            {"experts route + plan": (lambda: ex.experts_plan(logits, g, sc), T * (4 * g.experts + 8 * g.top)),
             "experts gather": (lambda: (ex.experts_plan(logits, g, sc), ex.experts_gather(h, g, sc)), 2 * 2 * T * g.top * d)})
    t.add("residual + experts' sum + norm", lambda: ops.stream_norm(x, d, y1=y, experts=sc.y[:T * g.top], expert_weights=sc.w[:T], weight=lw.norm1[0],
                                                                     eps=eps, h=h), T * d * (4 * 3 + 2 + 2 * g.top), 0)
    if r.loop_in is not None:
        t.gemm("loop entry", T, r.wp, 2 * r.wp, lambda: r._enter_pass(T), 4)
    if decode:
        lg = r.logits_padded[:T]
        t.gemm("head", T, r.vp, r.wp, lambda: r._head(r.hl[:T], lg), 4)
    return t.rows


def fogurax_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """The first layer of every kind of mixer, the experts, the token input and what joins them."""
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    d, eps, m = cfg.hidden_size, cfg.norm_eps, cfg.residual_mult
    x, h, y = r.x[:T], r.xb[:T], r.y[:T]
    h.normal_()
    b = r._decode_batch(T) if decode else _prompt_batch(r, T)
    seen = set()
    for run in r.runs:
        lw = run.layer
        kind = lw.spec.mixer.type
        if kind in seen:
            continue
        seen.add(kind)
        both = kind == "parallel"
        w, part, cache = (lw.mix.left, lw.mixer.left, run.cache[0]) if both else (lw.mix, lw.mixer, run.cache)
        g, plan = w.geo, part.planned(b)
        H, G, D, n = g.heads, g.kv_heads, g.dp, g.heads * g.dp
        proj, q = part._projected(w, T), part.q[:T * n].view(T, n)
        out = lw.mixer.out[:T * lw.mix.wo.shape[1]].view(T, -1)
        t.gemm(f"{kind}: joint projection", T, w.wproj.shape[0], r.wp, lambda: r._project(lw, h))
        small = r._project(lw, h)
        t.add(f"{kind}: norm + rotation + append", lambda: ops.grouped_append(
            proj, g, conv=w.conv, cache=cache, cu_q=b.cu_q, positions=b.positions, state_slots=b.state_slots, slots=b.slots, q_norm=w.q_norm,
            k_norm=w.k_norm, eps=eps, table=w.table, q=q), 2 * T * (g.channels * 2 + (g.history if decode else 0) * 2), 0)
        fn = lambda: ops.grouped_attention(q, g, cache, b.block_tables, b.cu_q, b.seq_lens, out[:, :n], scale=w.spec.scale, rows=T, max_q=b.max_new,
                                           n_single=b.n_single, gate=small if w.spec.form.gate else None, workspace=part.workspace, splits=plan.get(g, 1))
        reach = g.reach or max(context, T)
        if decode:
            span = (context - 1) % g.chunk + 1 if g.chunk else min(context, reach)
            t.add(f"{kind}: attention", fn, 2 * T * (2 * span * G * D + 2 * H * D), 4.0 * T * H * span * D)
        else:
            pairs = sum(i % g.chunk + 1 if g.chunk else min(i + 1, reach) for i in range(T))
            t.add(f"{kind}: attention", fn, 2 * T * D * (2 * H + 2 * G), 4.0 * pairs * H * D)
        if both:
            _time_mix_rows(t, r, lw.mixer.right, lw.mix.right, run.cache[1], h, out[:, n:], b, T, decode)
        t.gemm(f"{kind}: output projection", T, r.wp, out.shape[1], lambda: ops.gemm(out, lw.mix.wo, out=y, out_f32=True), 4)
    lw = r.layers[0]
    logits = r._project(lw, h)[:, lw.mix_small:]
    w, g = lw.ff, lw.ff.geo
    sc = lw.feed_forward.scratch[g]
    _routed(t, T, g.experts, g.top, d, g.ff, lambda: ex.experts_up(g, sc, w.wgu, T), lambda: ex.experts_down(g, sc, w.wd), None,
            {"experts route + plan": (lambda: ex.experts_plan(logits, g, sc), T * (4 * g.experts + 8 * g.top)),
             "experts gather": (lambda: (ex.experts_plan(logits, g, sc), ex.experts_gather(h, g, sc)), 2 * 2 * T * g.top * d)})
    shared = w.shared
    act = r._part(DensePart).act[:T * shared.ffp].view(T, shared.ffp)
    t.gemm("shared gate|up + unit", T, 2 * shared.ffp, r.wp, lambda: ops.gemm(h, shared.wgu, out=act, bn=256, swiglu=True), 2, shared.ffp)
    t.gemm("shared down", T, r.wp, shared.ffp, lambda: ops.gemm(act, shared.wd, out=r.y2[:T], out_f32=True), 4)
    t.add("residual + experts' sum", lambda: ops.stream_norm(x, d, y1=y, y2=r.y2[:T], experts=sc.y[:T * g.top], top=g.top, mult=m, copy=h),
          T * d * (4 * 4 + 2 + 2 * g.top), 0)
    z, a = r.side_z[:T], r.side_a[:T]
    t.gemm("token input: gate", T, r.sp, r.wp, lambda: ops.gemm(h, lw.side.gate, out=z, out_f32=True), 4)
    t.add("token input: unit", lambda: ops.token_side(z, b.tokens[:T], r.side_embed, 0, a, r.side_dim), T * r.side_dim * 8, 0)
    t.gemm("token input: projection", T, r.wp, r.sp, lambda: ops.gemm(a, lw.side.proj, out=y, out_f32=True), 4)
    t.add("token input's norm + residual + norm", lambda: ops.stream_norm(x, d, side=y, side_weight=lw.side.norm, mult=m, weight=lw.norm1[0], eps=eps, h=h),
          T * d * (4 * 3 + 2), 0)
    if decode:
        lg = r.logits_padded[:T]
        t.gemm("head", T, r.vp, r.wp, lambda: r._head(r.hl[:T], lg), 4)
    return t.rows


def sumitar_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """The first layer of every kind of mixer and feed-forward, and what joins them."""
    r, cfg, t = eng.runner, eng.runner.cfg, _Table()
    d, eps = cfg.hidden_size, cfg.norm_eps
    x, h, y, y2 = r.x[:T], r.xb[:T], r.y[:T], r.y2[:T]
    h.normal_()
    b = r._decode_batch(T) if decode else _prompt_batch(r, T)
    run = next(x for x in r.runs if x.layer.spec.mixer.type == "delta")
    lw, w, part, cache = run.layer, run.layer.mix, run.layer.mixer, run.cache
    g, plan = w.geo, part.planned(b)
    H, n = g.heads, g.heads * g.vp
    t.gemm("delta: joint projection", T, w.wproj.shape[0], r.wp, lambda: r._project(lw, h))
    small = r._project(lw, h)
    rows, rule = part.prepare(w, cache, small, b)
    t.add("delta: convolution + units", lambda: part.prepare(w, cache, small, b), 2 * T * g.channels * (2 + ((w.spec.taps - 1) * 2 if decode else 0)), 0)
    o, out = part.o[:T * n].view(T, n), part.out[:T * n].view(T, n)
    t.add("delta: recurrence", lambda: part.recur(w, cache, rows, rule, o, b, plan), T * (2 * g.channels + 4 * n) + 2 * 4 * H * g.kp * g.vp * b.rows,
          T * H * ((6.0 if decode else 8.0) * g.kp * g.vp + (0 if decode else 2.0 * 64 * (3 * g.kp + 2 * g.vp))))
    t.add("delta: norm + gate", lambda: ops.gated_norm(o, w.norm, part._projected(w, T)[:, g.offsets[3]:], g, eps, out, True, silu=True), T * n * 8, 0)
    t.gemm("delta: output projection", T, r.wp, n, lambda: ops.gemm(out, w.wo, out=y, out_f32=True), 4)

    run = next(x for x in r.runs if x.layer.spec.mixer.type == "parallel")
    pair, left, right = run.layer.mix, run.layer.mixer.left, run.layer.mixer.right
    w, g, plan = pair.left, pair.left.geo, left.planned(b)
    H, G, D, n = g.heads, g.kv_heads, g.dp, g.heads * g.dp
    t.gemm("parallel: joint projection", T, pair.wproj.shape[0], r.wp, lambda: r._project(run.layer, h))
    small = r._project(run.layer, h)
    proj = run.layer.mixer._projected(pair, T)
    q, out = left.q[:T * n].view(T, n), left.out[:T * n].view(T, n)
    t.add("parallel: rotation + append", lambda: ops.grouped_append(
        proj[:, pair.right.geo.proj:], g, conv=None, cache=run.cache[0], cu_q=b.cu_q, positions=b.positions, state_slots=b.state_slots, slots=b.slots,
        q_norm=None, k_norm=None, eps=eps, table=w.table, q=q, q_factor=w.temp), 2 * T * g.channels * 2, 0)
    fn = lambda: ops.grouped_attention(q, g, run.cache[0], b.block_tables, b.cu_q, b.seq_lens, out, scale=w.spec.scale, rows=T, max_q=b.max_new,
                                       n_single=b.n_single, workspace=left.workspace, splits=plan.get(g, 1))
    if decode:
        span = min(context, g.window)
        t.add("parallel: attention", fn, 2 * T * (2 * span * G * D + 2 * H * D), 4.0 * T * H * span * D)
    else:
        t.add("parallel: attention", fn, 2 * T * D * (2 * H + 2 * G), 4.0 * sum(min(i + 1, g.window) for i in range(T)) * H * D)
    t.gemm("parallel: output projection, attention", T, r.wp, n, lambda: ops.gemm(out, w.wo, out=y, out_f32=True), 4)
    rw, rg = pair.right, pair.right.geo
    m = rg.heads * rg.vp
    mixed = right.out[:T * m].view(T, m)
    t.add("parallel: forget mixing + norm", lambda: right.recur(rw, run.cache[1], proj, small, mixed, b, right.planned(b)),
          T * m * (2 * 3 + 4) + 2 * 4 * m * rg.kp * b.rows, T * rg.heads * (4.0 * rg.kp * rg.vp + (0 if decode else 2.0 * 64 * (rg.kp + rg.vp))))
    t.gemm("parallel: output projection, forget mixing", T, r.wp, m, lambda: ops.gemm(mixed, rw.wo, out=y2, out_f32=True), 4)
    norms = dict(post=lw.norm1b, pre=lw.norm2, eps=eps, h=h)
    t.add("halves' norms + residual + norm", lambda: ops.stream_sandwich(x, d, y=y, pair=(y2, pair.left_out, pair.right_out), **norms), T * d * (4 * 4 + 2), 0)
    t.add("norm + residual + norm", lambda: ops.stream_sandwich(x, d, y=y, **norms), T * d * (4 * 3 + 2), 0)

    lw = r.layers[0]
    w, act = lw.ff, lw.feed_forward
    z, a = act.z[:T * w.ffp].view(T, w.ffp), act.a[:T * w.ffp].view(T, w.ffp)
    t.gemm("dense: up", T, w.ffp, r.wp, lambda: ops.gemm(h, w.wu, out=z))
    t.add("dense: normed powers", lambda: ops.poly_norm(z, w.act, w.spec.ff, eps, a), T * w.ffp * 4, 0)
    t.gemm("dense: down", T, r.wp, w.ffp, lambda: ops.gemm(a, w.wd, out=y, out_f32=True), 4)
    lw = next(x for x in r.layers if x.spec.mlp.kind == "moe")
    small = r._small_rows(h, lw.wsmall_ff)
    e, g = lw.ff, lw.ff.geo
    sc = lw.feed_forward.scratch[g]
    t.gemm("router", T, lw.wsmall_ff.shape[0], r.wp, lambda: r._small_rows(h, lw.wsmall_ff), 4)
    _routed(t, T, g.experts, g.top, d, g.ff, lambda: ex.experts_up(g, sc, e.wgu, T), lambda: ex.experts_down(g, sc, e.wd), None,
            {"experts route + plan": (lambda: ex.experts_plan(small, g, sc, e.correction), T * (4 * g.choices + 8 * g.top)),
             "experts gather": (lambda: (ex.experts_plan(small, g, sc, e.correction), ex.experts_gather(h, g, sc)), 2 * 2 * T * g.top * d)})
    shared = e.shared
    act = r._part(DensePart).act[:T * shared.ffp].view(T, shared.ffp)
    t.gemm("shared gate|up + unit", T, 2 * shared.ffp, r.wp, lambda: ops.gemm(h, shared.wgu, out=act, bn=256, swiglu=True), 2, shared.ffp)
    t.gemm("shared down", T, r.wp, shared.ffp, lambda: ops.gemm(act, shared.wd, out=y, out_f32=True), 4)
    chosen = ops.ChosenExperts(sc.y[:T * g.top], sc.w[:T], sc.idx[:T], g.experts, h)
    t.add("experts' sum + norm + residual + norm", lambda: ops.stream_sandwich(x, d, y=y, gate=small[:, g.choices:], chosen=chosen, **norms),
          T * d * (4 * 3 + 2 + 2 * g.top), 0)
    if decode:
        lg = r.logits_padded[:T]
        t.gemm("head", T, r.vp, r.wp, lambda: r._head(r.hl[:T], lg), 4)
    return t.rows


def _time_mix_rows(t: _Table, r, part, w, cache, h, out, b, T: int, decode: bool) -> None:
    g, eps = w.geo, r.cfg.norm_eps
    n = g.heads * g.kp
    mixed, plan = part.mixed, part.planned(b)
    t.add("time mixing: shift", lambda: ops.token_shift(h, w.mu, mixed, cache.history, b.cu_q, b.positions, b.state_slots), 2 * T * r.wp * 6, 0)
    proj = part.project_mixes(w, T)
    t.gemm("time mixing: r, k, v, gate", T, 4 * n, r.wp, lambda: part.project_mixes(w, T))
    t.add("time mixing: decay's products", lambda: part.decay_logits(w, T), 2 * T * r.wp + 2 * w.rank * (r.wp + 2 * n) + 4 * T * n,
          2.0 * T * w.rank * (r.wp + 2 * n))
    z = part.decay_logits(w, T)
    state = 2 * 4 * n * g.vp
    t.add("time mixing: recurrence + norm + gate", lambda: part.recur(w, cache, proj, z, out, b, plan), T * n * (2 * 5 + 4) + state * b.rows,
          T * g.heads * (4.0 * g.kp * g.vp + (0 if decode else 2.0 * 64 * (g.kp + g.vp))))


def _prompt_batch(r, T: int):
    """One whole prompt of T tokens."""
    i32 = dict(dtype=torch.int32, device="cuda")
    pos = torch.arange(T, **i32)
    return type(r._decode_batch(2))(rows=1, num_tokens=T, padded=T, max_new=T, tokens=pos, positions=pos, slots=pos, cu_q=torch.tensor([0, T], **i32),
                                    seq_lens=torch.tensor([T], **i32), block_tables=torch.arange(-(-T // 16), **i32)[None].contiguous(),
                                    host_cu_q=[0, T], host_seq_lens=[T], state_slots=torch.zeros(1, **i32), n_single=0)


def hf_kernels(eng: InferenceEngine, T: int, context: int, decode: bool) -> dict:
    """The first layer of a Hugging Face style model (dense or routed experts)."""
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
    if lw.moe is not None:
        m = lw.moe
        h.normal_()
        m.forward(h, x)
        n = T * m.k
        t.add("experts layer, all launches", lambda: m.forward(h, x), 2 * (min(m.E, n) * 3 * m.F * d + 2 * T * d), 6.0 * n * d * m.F)
        t.gemm("router", T, m.E, d, lambda: ops.gemm(h, m.gate, out=m.logits[:T], out_f32=True), 4)
        _routed(t, T, m.E, m.k, d, m.F, lambda: m._grouped(m.xp, m.wgu, m.gu, 2 * m.F, d, m.BN_GU, m.tiles_gu, m.ntiles.data_ptr(), None),
                lambda: m._grouped(m.act, m.wd, None, d, m.F, m.BN_DN, m.tiles_dn, m.ntiles.data_ptr() + 4, m.ret),
                lambda: ops.swiglu(m.gu[:n], out=m.act[:n]))
    else:
        act = torch.empty(T, r.F, dtype=torch.bfloat16, device="cuda")
        t.gemm("gate|up + unit", T, 2 * r.F, d, lambda: ops.gemm(h, lw.wgu, out=act, bn=r.swiglu_bn, swiglu=True, norm_eps=fold), 2, r.F)
        t.gemm("down projection", T, d, r.F, lambda: ops.gemm(act, lw.wd, residual=x, out=x))
    if decode:
        t.gemm("head", T, cfg.vocab_size, d, lambda: ops.gemm(h, r.lm_head, out=r.a_logits[:T], out_f32=True), 4)
    return t.rows


# design -> (sizes, pair of configurations, labels and kernel tables)
DESIGNS = {"lulezen": (SIZES, configs, (("lulezen", latent_kernels), ("llama", hf_kernels))),
           "zamusun": (EXPERT_SIZES, expert_configs, (("zamusun", expert_stack_kernels), ("qwen3_moe", hf_kernels))),
           "fogurax": (EXPERT_SIZES, fogurax_configs, (("fogurax", fogurax_kernels), ("qwen3_moe", hf_kernels))),
           "sumitar": (EXPERT_SIZES, sumitar_configs, (("sumitar", sumitar_kernels), ("fogurax", fogurax_kernels)))}


def run(sizes: tuple[str, ...] = (), batches: tuple[int, ...] = (1, 64, 256), context: int = 2048, prompts: tuple[int, ...] = (512, 4096),
        kernels: bool = True, designs: tuple[str, ...] = ()) -> dict:
    out: dict = {"peaks": dict(zip(("hbm_bytes_s", "bf16_flop_s", "origin"), peaks())), "context": context, "sizes": {}}
    for design, (all_sizes, make, sides) in DESIGNS.items():
        if designs and design not in designs:
            continue
        for s in all_sizes:
            if sizes and s.name not in sizes:
                continue
            res: dict = {"shape": {k: v for k, v in s.__dict__.items() if k != "name"}}
            for (label, table), cfg in zip(sides, make(s)):
                res[label] = _measure(cfg, table, batches, context, prompts, kernels)
            out["sizes"][f"{design} {s.name}"] = res
    return out


def _measure(cfg, table, batches, context: int, prompts, kernels: bool) -> dict:
    one: dict = {"params_m": round(cfg.num_params() / 1e6), "decode": {}, "prefill": {}, "decode_kernels": {}, "prefill_kernels": {}}
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
    return one

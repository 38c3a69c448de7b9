"""The Sumitar design in the framework against the plain oracle (``sumitar_oracle.py``): whole prompts, portions, decoding, mixed
batches, state slots and blocks that are used again, greedy generation through the scheduler, trace replay.

Every engine test runs on the CPU twins of the ops (fp32) and, on a GPU, in both number formats. Random weights are scaled so
that attention is peaked, decays keep what is far back, and every mechanism moves the logits; ``test_oracle_mistakes_show`` plants
mistakes in the oracle and checks that each is far outside the tolerances used here.
"""

import json
import math
import os
import subprocess

import pytest
import sumitar_oracle as oracle
import torch
from test_lulezen import cut, feed_all, read_f32, tokens_for, trace_lines

from research_b200.inference import EngineConfig, InferenceEngine, SamplingParams
from research_b200.inference.trace_replay import make_engine, replay
from research_b200.models import config_from_dict, get_preset, init_random_weights, load_config, load_safetensors_dir, save_safetensors_dir
from research_b200.models.stack import DeltaRuleSpec, LayerStackConfig, NormedPairSpec

PLACES = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
TOL = {"float32": 3e-5, "bfloat16": 0.08}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def both(heads=4, kv_heads=2, dim=24, vdim=40, rot=12, base=3e4, size=29, mix=(3, 20, 36), scale=None):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                                   "rot": {"base": base, "dims": rot}, "scale": 2.5 * dim ** -0.5 if scale is None else scale},
                                          "right": dict(zip(("heads", "dim", "vdim"), mix))}}


def delta(heads=4, kv_heads=2, dim=24, vdim=20, taps=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def routed(experts=5, identity=2, top=3, ff=40, shared=56):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff}, "shared": {"ff": shared}}


def model(layers, vocab=130, width=56, eps=1e-5):
    return {"architecture": "Sumitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [{**m, "mlp": f} for m, f in layers]}


CONFIGS = {
    "mixed": model([(delta(), routed()), (both(), dense()), (delta(6, 2, 32, 24, 4), None), (both(2, 1, 20, 20, 8, 1e4, 60, (2, 40, 40)), routed(7, 1, 4, 24, 16))]),
    "ones": model([(both(1, 1, 10, 9, 4, 50.0, 1, (1, 9, 1)), routed(1, 1, 1, 17, 8)), (delta(1, 1, 10, 7, 1), None), (delta(1, 1, 1, 12, 2), dense(9))],
                  vocab=61, width=30, eps=1e-3),
    "wide": model([(both(20, 1, 128, 72, 100, 1e5, 70, (2, 64, 64)), routed(9, 3, 4, 200, 130)), (delta(4, 4, 128, 128, 4), dense(300)),
                   (delta(2, 1, 64, 192, 2), None), (both(3, 3, 80, 112, 20, 1e4, 130, (1, 100, 128)), dense(90))], vocab=97, width=72),
    "odd": model([(delta(2, 2, 150, 60, 6), None), (both(2, 2, 30, 200, 30, 1e4, 50, (2, 33, 150)), dense(33)), (delta(3, 1, 40, 136, 9), routed(3, 4, 5))],
                 vocab=83, width=46),
}


def weights_for(name, seed=0, c=None):
    """Random weights that make every part count: peaked scores, decays between nothing and nearly everything, uneven norms, corrections that
    decide. All values are exact in bf16, so that both number formats and the oracle see the same model."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for key, shape in config_from_dict(CONFIGS[name] if c is None else c).param_shapes().items():
        last = key.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "alpha":
            t = 0.5 + 0.2 * r.abs()
        elif key.endswith(".f.b"):
            t = 3.0 * r + 3.0
        elif last == "b" and len(shape) == 1:
            t = (0.2 if "norm" in key else 0.5) * r
        elif last == "lower":
            t = (torch.rand(shape, generator=g) * 1.6 - 0.7).clamp(min=0)
        elif last == "A_log":
            t = 1.5 * r - 1.0
        elif last == "dt_bias":
            t = 1.5 * r - 3.0
        elif last in ("temp", "out") or last.startswith("norm"):
            t = 0.3 * r + 1.0
        elif last == "correction":
            t = 0.6 * r.abs()
        elif last == "act":
            t = torch.tensor([0.6, -0.4, 0.5, 0.2])
        elif last == "conv":
            t = 0.6 * r
        else:
            gain = {"q": 2.0, "k": 1.5, "router": 4.0, "gate": 1.5, "up": 1.5, "f": 1.5, "b": 2.0, "a": 1.5, "sg": 2.0}.get(last, 1.0)
            t = r * (1.0 if key == "embed" else gain / math.sqrt(shape[1]))
        out[key] = t.bfloat16()
    return out


_CACHE = {}


def wanted(name, tokens):
    """Oracle logits in float64, remembered per prompt."""
    key = (name, tuple(tokens))
    if key not in _CACHE:
        _CACHE[key] = oracle.forward(tokens, {k: v.double() for k, v in weights_for(name).items()}, CONFIGS[name])
    return _CACHE[key]


def errors(got, want):
    """rms difference of every row, relative to the spread of the expected logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()


def agree(got, want, dtype):
    """All rows within the tolerance. In bf16 two experts may score so nearly alike that rounding picks the other one: one row
    in twenty may be further off."""
    e = errors(got, want)
    if dtype == "bfloat16":
        e = e.sort().values[:len(e) - len(e) // 20]
    assert e.max() < TOL[dtype], e.max()


def engine(name, place, **kw):
    opts = dict(cache_type="none", max_batch_size=4, max_model_len=480, max_tokens_per_batch=480, num_kv_blocks=64, ignore_eos=True,
                dtype=place[1], graph_batch_sizes=(1, 2, 4))
    opts.update(kw)
    return InferenceEngine(EngineConfig(**opts), config_from_dict(CONFIGS[name]), weights_for(name), device=place[0])


# ------------------------------------------------------------------------------------------ configuration and weights
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_and_checkpoint(name, tmp_path):
    c = CONFIGS[name]
    cfg = config_from_dict(c)
    assert isinstance(cfg, LayerStackConfig) and config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert cfg.tie_word_embeddings and [x.mixer.type for x in cfg.layers] == [e["type"] for e in c["layers"]]
    w = weights_for(name)
    assert "head" not in w and w["final.norm.alpha"].shape == () and ("l0.norm2b.b" in w) == (c["layers"][0]["mlp"] is not None)
    save_safetensors_dir(w, cfg, tmp_path)
    back, cfg2 = load_safetensors_dir(tmp_path)
    assert cfg2 == cfg == load_config(tmp_path) and all(torch.equal(back[k], v) for k, v in w.items())
    assert {k: tuple(v.shape) for k, v in back.items()} == cfg.param_shapes()
    r = init_random_weights(cfg, seed=3)
    assert (r["l0.norm1"] == 1).all() and (r["l0.norm1b.b"] == 0).all() and cfg.num_params() == sum(t.numel() for t in r.values())
    for i, e in enumerate(c["layers"]):
        if e["type"] == "delta":
            assert r[f"l{i}.mix.b"].abs().max() > 0


def test_presets_and_limits():
    cfg = get_preset("tiny-sumitar")
    assert [type(x.mixer) for x in cfg.layers] == [NormedPairSpec, DeltaRuleSpec, DeltaRuleSpec] and cfg.layers[1].mlp.identity == 3
    assert 3.5e9 < get_preset("sumitar-4b").num_params() < 5.0e9
    for bad, what in ((model([(delta(dim=600), None)]), "key channels"), (model([(delta(vdim=600), None)]), "value channels"),
                      (model([(delta(taps=17), None)]), "convolutions"), (model([(both(dim=600), None)]), "channels"),
                      (model([(both(mix=(1, 20, 600)), None)]), "key channels"), (model([(delta(), routed(250, 10))]), "experts")):
        with pytest.raises(ValueError, match=what):
            InferenceEngine(EngineConfig(max_batch_size=2, max_model_len=64, num_kv_blocks=8), config_from_dict(bad), weights_for("", c=bad), device="cpu")
    with pytest.raises(ValueError, match="unknown mixer"):
        config_from_dict({**CONFIGS["mixed"], "layers": [{"type": "mlstm", "mixer": {}, "mlp": None}]})


@pytest.mark.parametrize("place", PLACES)
def test_without_identities_or_a_shared_expert(place):
    """Routers of experts alone, written with and without the keys that are zero."""
    f = routed(4, 0, 2, 24)
    c = model([(delta(2, 1, 16, 16, 2), {**f, "shared": None}), (both(2, 1, 16, 16, 8, mix=(1, 8, 8)), {**f, "router": {"experts": 4, "top": 2}})], vocab=50, width=32)
    w = weights_for("", 4, c)
    assert "l0.mlp.shared.sg" not in w and w["l1.mlp.router"].shape[0] == 4
    eng = InferenceEngine(EngineConfig(cache_type="none", max_batch_size=2, max_model_len=128, num_kv_blocks=16, dtype=place[1], graph_batch_sizes=(1, 2)),
                          config_from_dict(c), w, device=place[0])
    toks = tokens_for(c, 60, 3)
    agree(feed_all(eng, toks, [40] + [1] * 20), oracle.forward(toks, {k: v.double() for k, v in w.items()}, c), place[1])


def test_oracle_mistakes_show(monkeypatch):
    """The tolerances can tell: every mechanism left out or off by a little moves the logits far more."""
    name = "mixed"
    c = CONFIGS[name]
    toks = tokens_for(c, 120, 5)
    w = {k: v.double() for k, v in weights_for(name).items()}
    right = oracle.forward(toks, w, c)

    def wrong(config=None, weights=None, **patched):
        c2, w2 = json.loads(json.dumps(c)), dict(w)
        if config:
            config(c2)
        if weights:
            weights(w2)
        with monkeypatch.context() as m:
            for k, f in patched.items():
                m.setattr(oracle, k, f)
            return errors(oracle.forward(toks, w2, c2), right).quantile(0.95).item()

    def scaled(name, by):
        return lambda x: x.update({name: x[name] * by})

    def mixer(x, i):
        return x["layers"][i]["mixer"]

    seen_window, rms, route = oracle.seen_window, oracle.rms, oracle.route

    def no_write_gate(q, f, v):
        S, out = 0, []
        for i in range(len(q)):
            S = f[i][:, :, None] * S + v[i][:, None, :]
            out.append(torch.einsum("hde,hd->he", S, q[i]))
        return torch.stack(out)

    def read_first(q, k, v, g, beta):
        S, out = v.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
        for i in range(len(q)):
            out.append(torch.einsum("hde,hd->he", S, q[i]))
            S = g[i][:, None, None] * S
            u = beta[i][:, None] * (v[i] - torch.einsum("hde,hd->he", S, k[i]))
            S = S + k[i][:, :, None] * u[:, None, :]
        return torch.stack(out)

    def no_correction(q, k, v, g, beta):
        S, out = v.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
        for i in range(len(q)):
            S = g[i][:, None, None] * S + k[i][:, :, None] * (beta[i][:, None] * v[i])[:, None, :]
            out.append(torch.einsum("hde,hd->he", S, q[i]))
        return torch.stack(out)

    got = {
        "bias": wrong(weights=scaled("l1.mix.left.k.b", 0)),
        "temperature": wrong(weights=lambda x: x.update({"l1.mix.left.temp": torch.ones(4, dtype=torch.float64)})),
        "no rotation": wrong(rotate=lambda x, rot: x),
        "no window": wrong(seen_window=lambda t, size: seen_window(t, 1000)),
        "window": wrong(seen_window=lambda t, size: seen_window(t, size + 1)),
        "left": wrong(weights=scaled("l1.mix.left.out", 1.5)),
        "right": wrong(weights=scaled("l1.mix.right.out", 1.5)),
        "halves' norm": wrong(MIXERS={**oracle.MIXERS, "parallel": lambda h, w, n, m, e: (
            oracle.window_attention(h, w, n + ".left", m["left"]) * w[n + ".left.out"]
            + oracle.forget_mix(h, w, n + ".right", m["right"], e) * w[n + ".right.out"]) / 2}),
        "lower bound": wrong(weights=scaled("l3.mix.right.lower", 0)),
        "write gate": wrong(forget_scan=no_write_gate),
        "forget state": wrong(forget_scan=lambda q, f, v: torch.einsum("thd,thd,the->the", q, 1 - f, v)),
        "forget bias": wrong(weights=scaled("l1.mix.right.f.b", 0)),
        "conv": wrong(causal_conv=lambda u, t: u * t[:, -1]),
        "conv turned": wrong(causal_conv=lambda u, t, f=oracle.causal_conv: f(u, t.flip(1))),
        "unit": wrong(unit=lambda x: x),
        "reads first": wrong(delta_scan=read_first),
        "no delta": wrong(delta_scan=no_correction),
        "step size": wrong(delta_scan=lambda q, k, v, g, b, f=oracle.delta_scan: f(q, k, v, g, torch.ones_like(b))),
        "decay": wrong(delta_scan=lambda q, k, v, g, b, f=oracle.delta_scan: f(q, k, v, torch.ones_like(g), b)),
        "decay's bias": wrong(weights=scaled("l0.mix.dt_bias", 0)),
        "groups": wrong(lambda x: mixer(x, 0).update(kv_heads=4), weights=lambda x: x.update({f"l0.mix.{s}{e}": x[f"l0.mix.{s}{e}"].repeat(2, 1)
                                                                                             for s in "qk" for e in ("", ".conv")})),
        "polynomial": wrong(poly_norm=lambda z, act, eps: act[0] * rms(z, eps) + act[3]),
        "e": wrong(weights=lambda x: x.update({"l1.mlp.act": x["l1.mlp.act"] * torch.tensor([1, 1, 1, 0.0], dtype=torch.float64)})),
        "correction": wrong(route=lambda z, corr, top: route(z, 0 * corr, top)),
        "corrected weights": wrong(route=lambda z, corr, top: (route(z, corr, top)[0], torch.gather(torch.softmax(z, -1) + corr, -1, route(z, corr, top)[0]))),
        "renormalized": wrong(route=lambda z, corr, top: (route(z, corr, top)[0], route(z, corr, top)[1] / route(z, corr, top)[1].sum(-1, keepdim=True))),
        "identity": wrong(lambda x: [e["mlp"]["router"].update(identity=0) for e in x["layers"] if e["mlp"] and e["mlp"]["kind"] == "moe"]),
        "shared gate": wrong(weights=scaled("l0.mlp.shared.sg", 0)),
        "shared": wrong(weights=scaled("l0.mlp.shared.down", 0)),
        "alpha": wrong(weights=scaled("l0.norm1b.alpha", 1.1)),
        "norm's bias": wrong(weights=scaled("l2.norm1b.b", 0)),
        "final": wrong(weights=scaled("final.norm.alpha", 1.1)),
        "eps": wrong(rms=lambda v, eps: rms(v, eps + 1e-3)),
    }
    # (what only stretches or weighs a part of some heads moves less; the exact mode tells it by far)
    fine = {"bias", "temperature", "window", "eps", "left", "right", "alpha", "norm's bias", "final", "decay's bias", "lower bound", "shared gate", "e",
            "forget bias", "corrected weights", "decay"}
    small = {k: v for k, v in got.items() if v < (100 * TOL["float32"] if k in fine else 1.5 * TOL["bfloat16"])}
    assert not small, small


# ------------------------------------------------------------------------------------------ logits through the engine
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_portions_and_single_tokens(name, place):
    toks = tokens_for(CONFIGS[name], 290, 5)
    want = wanted(name, toks)
    eng = engine(name, place)
    for portions in ([290], cut(290, 37), cut(290, 2) if name == "mixed" else cut(290, 130), [1, 128, 3, 16, 17, 125],
                     [5] + [1] * 20 + [140] + [1] * 15 + [110]):
        agree(feed_all(eng, toks, portions), want, place[1])
    assert eng.check_invariants() == 0 and eng.cache_stats()["free_blocks"] == 64


@pytest.mark.parametrize("place", PLACES)
def test_unequal_requests_in_one_batch_and_reused_slots(place):
    """Portions beside single tokens, requests that pause, blocks and state slots that only fit the live ones: rows equal the
    request alone."""
    name = "mixed"
    prompts = {k: tokens_for(CONFIGS[name], n, 20 + i) for i, (k, n) in enumerate({"a": 190, "b": 40, "c": 1, "d": 170, "e": 160, "f": 90}.items())}
    eng = engine(name, place, num_kv_blocks=28)
    steps = [{"a": 130, "b": 2, "c": 1}, {"a": 1, "b": 20, "d": 133}, {"a": 1, "d": 2}, {"a": 20, "b": 1, "d": 1}, {"b": 17, "a": 2},
             {"a": 36, "d": 34}, {"e": 3, "f": 50}, {"e": 1, "f": 1}, {"f": 39, "e": 156}]
    at, streams = dict.fromkeys(prompts, 0), {}
    got, want = [], []
    for step in steps:
        entries = []
        for k, n in step.items():
            if k not in streams:
                streams[k] = eng.open_stream()
            entries.append((streams[k], prompts[k][at[k]:at[k] + n], list(range(n))))
            want += [wanted(name, prompts[k])[p] for p in range(at[k], at[k] + n)]
            at[k] += n
        got.append(eng.feed(entries).cpu())
        assert eng.check_invariants() == 0
        for k in step:
            if at[k] == len(prompts[k]):
                eng.close_stream(streams[k])
    agree(torch.cat(got), torch.stack(want), place[1])
    assert all(at[k] == len(p) for k, p in prompts.items())
    assert eng.cache_stats()["free_blocks"] == 28 and eng.check_invariants() == 0


@pytest.mark.parametrize("place", PLACES)
def test_a_used_slot_starts_anew(place):
    """A request's rows are the same in a fresh engine and in slots and blocks that another request has filled."""
    name = "wide"
    eng = engine(name, place, max_batch_size=2, graph_batch_sizes=(1, 2))
    a, b = tokens_for(CONFIGS[name], 150, 1), tokens_for(CONFIGS[name], 140, 2)
    for portions in ([140], [1] * 12 + [128], cut(140, 15)):
        first = feed_all(eng, b, portions)
        feed_all(eng, a, [150])
        assert torch.equal(feed_all(eng, b, portions), first)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("kind,reach", [("delta", None), ("both", None), ("window", 45)])
def test_how_far_a_token_reaches(place, kind, reach):
    """One mixer, one changed token: nothing before it moves; what sees it does, across blocks, chunks and portions, and what does not
    see it stays (the window with the other half turned off)."""
    mix = {"delta": delta(2, 1, 16, 16, 3), "both": both(2, 1, 16, 16, 8, 1e4, 45, (2, 16, 24), scale=0.3),
           "window": both(2, 1, 16, 16, 8, 1e4, 45, (2, 16, 16), scale=0.05)}[kind]
    c = model([(mix, None)], vocab=50)
    w = weights_for("", 3, c)
    w.update({k: torch.full_like(v, 9.0) for k, v in w.items() if k.endswith("f.b")})       # states that keep all
    w.update({k: torch.full_like(v, -9.0) for k, v in w.items() if k.endswith("A_log")})
    if kind == "window":
        w["l0.mix.right.out"] = w["l0.mix.right.out"] * 0
    eng = InferenceEngine(EngineConfig(cache_type="none", max_batch_size=2, max_model_len=288, max_tokens_per_batch=288, num_kv_blocks=20,
                                       dtype=place[1], graph_batch_sizes=(1, 2)), config_from_dict(c), w, device=place[0])
    toks = tokens_for(c, 270, 9)
    for mark in (0, 15, 59, 60, 127, 128, 200):
        end = mark + reach if reach else 270
        other = list(toks)
        other[mark] = (toks[mark] + 7) % 50
        for portions in ([270], [3, 141] + [1] * 126, cut(270, 45)):
            moved = (feed_all(eng, toks, portions) - feed_all(eng, other, portions)).abs().amax(-1)
            assert (moved[:mark] == 0).all() and (moved[end:] == 0).all(), (mark, portions)
            assert (moved[mark:end] > 0).float().mean() > (0.98 if place[1] == "float32" else 0.8), (mark, portions)


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding(place):
    name = "mixed"
    toks = tokens_for(CONFIGS[name], 420, 31)
    agree(feed_all(engine(name, place), toks, [20] + [1] * 400), wanted(name, toks), place[1])


# ------------------------------------------------------------------------------------------ generation and scheduling
def check_greedy(name, prompt, sample, dtype):
    """fp32: the oracle's own greedy tokens. bf16: every chosen token is near the oracle's best, and its log-prob agrees."""
    w = {k: v.double() for k, v in weights_for(name).items()}
    ids = list(prompt) + list(sample.completion_tokens)
    lp = torch.log_softmax(oracle.forward(ids, w, CONFIGS[name])[len(prompt) - 1:-1], -1)
    tol = 5e-3 if dtype == "float32" else 2.5
    for row, tok, got in zip(lp, sample.completion_tokens, sample.logprobs):
        assert row[tok] > row.max() - tol and abs(row[tok] - got) < tol


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("cache,chunk", [("none", 0), ("radix", 13)])
def test_greedy_generation(place, cache, chunk):
    """A model whose layers keep state shares no prefixes, whatever cache is asked for."""
    name = "mixed"
    shared = tokens_for(CONFIGS[name], 40, 50)
    prompts = [shared + tokens_for(CONFIGS[name], n, 60 + n) for n in (3, 30, 117)] + [tokens_for(CONFIGS[name], n, 80 + n) for n in (1, 2, 60)]
    eng = engine(name, place, cache_type=cache, prefill_chunk=chunk, num_kv_blocks=80)
    for _ in range(2):
        for p, s in zip(prompts, eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9))):
            assert s.prompt_tokens == tuple(p) and len(s.completion_tokens) == 9 and s.cached_tokens == 0
            check_greedy(name, p, s, place[1])
    assert eng.check_invariants() == 0 and not eng.has_pending() and eng.cache_stats()["free_blocks"] == 80


@pytest.mark.parametrize("place", PLACES)
def test_prompt_longer_than_a_step_and_preemption(place):
    """A prompt beyond the step's token budget goes in portions beside decoding rows; a pool too small for all preempts, and a
    preempted request starts over in whatever slot it gets."""
    name = "mixed"
    prompts = [tokens_for(CONFIGS[name], n, 90 + n) for n in (150, 20, 33, 75)]
    eng = engine(name, place, max_tokens_per_batch=40, num_kv_blocks=17)
    joint = []
    step = eng._step_with_ids

    def watch():
        r = step()
        joint.append(eng.last_step_rows)
        assert eng.check_invariants() == 0
        return r

    eng._step_with_ids = watch
    for p, s in zip(prompts, eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=25))):
        assert len(s.completion_tokens) == 25
        check_greedy(name, p, s, place[1])
    assert any(a and b for a, b in joint), "no step mixed portions with decoding rows"
    assert eng.check_invariants() == 0 and eng.cache_stats()["free_blocks"] == 17


@pytest.mark.parametrize("place", PLACES)
def test_sampling_score_and_weight_update(place):
    name = "mixed"
    eng = engine(name, place, num_kv_blocks=80)
    p = [tokens_for(CONFIGS[name], 25, 1), tokens_for(CONFIGS[name], 140, 2)]
    a = eng.generate(p, SamplingParams(temperature=1.0, max_tokens=6, seed=7))
    b = eng.generate(p, SamplingParams(temperature=1.0, max_tokens=6, seed=7))
    assert [s.completion_tokens for s in a] == [s.completion_tokens for s in b]
    live = eng.open_stream()
    eng.feed([(live, p[0][:20], [])])
    agree(eng.runner.score(torch.tensor(p[1])), wanted(name, p[1]), place[1])     # scoring leaves live state alone
    agree(eng.feed([(live, p[0][20:], list(range(5)))]), wanted(name, p[0])[20:], place[1])
    eng.close_stream(live)
    w2 = weights_for(name, seed=9)
    eng.update_weights(w2)
    want = oracle.forward(p[1], {k: v.double() for k, v in w2.items()}, CONFIGS[name])
    s = eng.open_stream()
    assert errors(eng.feed([(s, p[1], list(range(140)))]), want).median() < TOL[place[1]]


def test_http_front_end_serves_it():
    from fastapi.testclient import TestClient

    from research_b200.inference.server import EngineService, create_app

    name = "mixed"
    svc = EngineService(engine(name, ("cpu", "float32"), num_kv_blocks=80))
    try:
        client = TestClient(create_app(svc, name))
        ids = tokens_for(CONFIGS[name], 30, 4)
        r = client.post("/generate", json={"input_ids": ids, "sampling_params": {"temperature": 0.0, "max_new_tokens": 5}}).json()
        assert [int(wanted(name, ids + r["output_ids"][:k])[-1].argmax()) for k in range(5)] == r["output_ids"]
    finally:
        svc.shutdown()


# ------------------------------------------------------------------------------------------ trace replay
def test_trace_replay_on_the_twins(tmp_path):
    name = "mixed"
    prompts = [tokens_for(CONFIGS[name], n, n) for n in (70, 30, 64)]
    save_safetensors_dir(weights_for(name), config_from_dict(CONFIGS[name]), tmp_path / "m")
    eng = make_engine(str(tmp_path / "m"), "float32", 112, device="cpu")
    lines, rows = trace_lines(prompts)
    done = []
    replay(eng, lines, tmp_path, done.append)
    by = dict(zip("abc", prompts))
    for i, want in enumerate(rows):
        agree(read_f32(tmp_path / f"{i}.f32", 130), torch.stack([wanted(name, by[k])[p] for k, p in want]), "float32")
    assert done == [0, 1, 2, 3] and eng.cache_stats()["free_blocks"] == 7


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(tmp_path, dtype, cuda_device):
    name = "wide"
    prompts = [tokens_for(CONFIGS[name], n, n) for n in (70, 30, 64)]
    save_safetensors_dir(weights_for(name), config_from_dict(CONFIGS[name]), tmp_path / "m")
    lines, rows = trace_lines(prompts)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "112"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    by = dict(zip("abc", prompts))
    for i, want in enumerate(rows):
        e = errors(read_f32(tmp_path / f"{i}.f32", 97), torch.stack([wanted(name, by[k])[p_] for k, p_ in want]))
        assert e.median() < TOL[dtype]

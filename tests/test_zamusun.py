"""The Zamusun design in the framework against the plain oracle (``zamusun_oracle.py``): whole prompts, portions, decoding, mixed
batches, state slots and blocks that are used again, greedy generation through the scheduler, trace replay.

Every engine test runs on the CPU twins of the ops (fp32) and, on a GPU, in both number formats. Random weights are scaled so
that attention is peaked, gates and decays keep what is far back, and every mechanism moves the logits;
``test_oracle_mistakes_show`` plants mistakes in the oracle and checks that each is far outside the tolerances used here.
"""

import json
import math
import os
import subprocess

import pytest
import torch
import zamusun_oracle as oracle
from test_lulezen import cut, feed_all, read_f32, tokens_for, trace_lines

from research_b200.inference import EngineConfig, InferenceEngine, SamplingParams
from research_b200.inference.trace_replay import make_engine, replay
from research_b200.models import config_from_dict, get_preset, init_random_weights, load_config, load_safetensors_dir, save_safetensors_dir
from research_b200.models.stack import LayerRun, LayerStackConfig

PLACES = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
TOL = {"float32": 3e-5, "bfloat16": 0.08}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def memory(heads=3, dim=24, vdim=20, cap=6.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def linear(heads=5, dim=12, vdim=40, slow=0.995):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                           "decay": [slow - (slow - 0.55) * h / max(heads - 1, 1) for h in range(heads)]}}


def attention(heads=6, kv_heads=2, dim=24, coef=0.4, every=16, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                                           "q_temp": {"coef": coef, "every": every}, "scale": dim ** -0.5 if scale is None else scale}}


def routed(experts=5, top=2, ff=40, limit=1.5):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def model(layers, vocab=130, width=56, eps=1e-5, loop=None):
    c = {"architecture": "Zamusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [{**m, "mlp": f} for m, f in layers]}
    return {**c, "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]}} if loop else c


CONFIGS = {
    "mixed": model([(memory(), routed()), (linear(), None), (attention(), routed(7, 3, 24, 0.8)), (memory(2, 40, 12, 4.0), None)], loop=(1, 3, 2)),
    "ones": model([(memory(1, 10, 9, 1.0), routed(1, 1, 17, 0.7)), (attention(1, 1, 10, 1.0, 1), None), (linear(1, 5, 7), routed(3, 1, 8, 3.0))],
                  vocab=61, width=30, eps=1e-3, loop=(0, 1, 1)),
    "wide": model([(attention(20, 1, 128, 0.2, 50), routed(9, 4, 200, 2.0)), (memory(2, 128, 128, 15.0), routed(9, 4, 200, 2.0)),
                   (linear(2, 80, 136), routed(4, 4, 16, 1.0))], vocab=97, width=72, loop=(1, 3, 3)),
    "odd": model([(attention(4, 4, 136, 0.3, 9, 0.05), None), (linear(2, 300, 24), routed()), (memory(2, 200, 130), None)], vocab=83, width=48),
}
RUNS = {"mixed": [0, 1, 2, 1, 2, 3], "ones": [0, 1, 2], "wide": [0, 1, 2, 1, 2, 1, 2], "odd": [0, 1, 2]}


def weights_for(config, seed=0):
    """Random weights that make every part count: peaked scores, sinks of a few units, forget gates that stay open for a
    while, uneven norms, clear routing. All values are exact in bf16, so that both number formats and the oracle see the same
    model."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in config_from_dict(config).param_shapes().items():
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "sink":
            t = 1.5 * r + 1.0
        elif name.endswith(".f.b"):
            t = r + 3.0
        elif last == "b":
            t = 0.5 * r
        elif last.startswith("norm"):
            t = 0.3 * r + (1.0 if ".mix." in name else 0.0)
        else:
            gain = {"q": 2.0, "k": 1.5, "router": 5.0, "gate": 1.5, "up": 1.5, "o": 0.7, "down": 1.0}.get(last, 1.0)
            t = r * (1.0 if name == "embed" else gain / math.sqrt(shape[1]))
        out[name] = t.bfloat16()
    return out


_CACHE = {}


def wanted(name, tokens):
    """Oracle logits in float64, remembered per prompt."""
    key = (name, tuple(tokens))
    if key not in _CACHE:
        w = {k: v.double() for k, v in weights_for(CONFIGS[name]).items()}
        _CACHE[key] = oracle.forward(tokens, w, CONFIGS[name])
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
    return InferenceEngine(EngineConfig(**opts), config_from_dict(CONFIGS[name]), weights_for(CONFIGS[name]), device=place[0])


# ------------------------------------------------------------------------------------------ configuration and weights
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_and_checkpoint(name, tmp_path):
    c = CONFIGS[name]
    cfg = config_from_dict(c)
    assert isinstance(cfg, LayerStackConfig) and config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert [r.layer for r in cfg.runs] == RUNS[name] == [i for i, _ in oracle.layer_order(c)]
    assert [r.enters for r in cfg.runs] == [e for _, e in oracle.layer_order(c)]
    w = weights_for(c)
    assert ("loop.in" in w) == ("loop" in c) and "head" not in w and "l0.norm2" not in w and "final.norm.b" not in w
    save_safetensors_dir(w, cfg, tmp_path)
    back, cfg2 = load_safetensors_dir(tmp_path)
    assert cfg2 == cfg == load_config(tmp_path) and all(torch.equal(back[k], v) for k, v in w.items())
    r = init_random_weights(cfg, seed=3)
    assert r["l0.norm1"].abs().max() == 0 and cfg.num_params() == sum(t.numel() for t in r.values())


def test_presets_and_limits():
    cfg = get_preset("tiny-zamusun")
    assert cfg.runs == (LayerRun(0, False), LayerRun(1, True), LayerRun(2, False), LayerRun(1, True), LayerRun(2, False))
    assert get_preset("zamusun-4b").tie_word_embeddings
    for bad, what in ((model([(attention(dim=600), None)]), "channels"), (model([(memory(dim=600), None)]), "key channels"),
                      (model([(linear(), routed(300, 2))]), "experts")):
        with pytest.raises(ValueError, match=what):
            InferenceEngine(EngineConfig(max_batch_size=2, max_model_len=64, num_kv_blocks=8), config_from_dict(bad), weights_for(bad), device="cpu")


def test_oracle_mistakes_show(monkeypatch):
    """The tolerances can tell: every mechanism left out or off by a little moves the logits far more."""
    name = "mixed"
    c = CONFIGS[name]
    toks = tokens_for(c, 120, 5)
    w = {k: v.double() for k, v in weights_for(c).items()}
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

    least = 1.5 * TOL["bfloat16"]
    assert wrong(weights=lambda x: x.update({"l2.mix.sink": x["l2.mix.sink"] - 1e4})) > least
    assert wrong(weights=lambda x: x.update({"l2.mix.k.b": x["l2.mix.k.b"] * 0})) > least
    assert wrong(weights=lambda x: x.update({"l0.mix.f.b": x["l0.mix.f.b"] * 0})) > least
    assert wrong(weights=lambda x: x.update({"l0.norm1": x["l0.norm1"] * 0})) > least
    assert wrong(weights=lambda x: x.update({"loop.in": x["loop.in"].roll(56, 1)})) > least
    assert wrong(lambda x: x["layers"][2]["mixer"]["q_temp"].update(coef=0.0)) > least
    assert wrong(lambda x: x["layers"][1]["mixer"].update(decay=[0.9] * 5)) > least
    assert wrong(lambda x: x["layers"][0]["mixer"].update(gate_cap=1.5)) > least
    assert wrong(lambda x: x["layers"][2]["mlp"]["expert"].update(limit=1e9)) > least
    assert wrong(lambda x: x["layers"][2]["mlp"]["router"].update(top=1)) > least
    assert wrong(lambda x: x["loop"].update(times=3)) > least
    assert wrong(silu=lambda z: z) > least
    assert wrong(route=lambda z, top: (torch.topk(z, top).indices, torch.full((*z.shape[:-1], top), 1 / top, dtype=z.dtype))) > TOL["bfloat16"]


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
    held = [eng.open_stream() for _ in range(5)]
    eng.feed([(s, [1, 2], []) for s in held[:4]])
    with pytest.raises(RuntimeError, match="state slot"):
        eng.feed([(held[4], [1, 2], [])])
    eng.close_stream(held[1])
    eng.feed([(held[4], [1, 2], [])])
    assert eng.check_invariants() == 0


@pytest.mark.parametrize("place", PLACES)
def test_a_used_slot_starts_from_zero(place):
    """A request's rows are the same in a fresh engine and in slots and blocks that another request has filled."""
    name = "wide"
    eng = engine(name, place, max_batch_size=2, graph_batch_sizes=(1, 2))
    a, b = tokens_for(CONFIGS[name], 150, 1), tokens_for(CONFIGS[name], 140, 2)
    for portions in ([140], [1] * 12 + [128], cut(140, 15)):
        first = feed_all(eng, b, portions)
        feed_all(eng, a, [150])
        assert torch.equal(feed_all(eng, b, portions), first)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("kind", ["memory", "linear", "attention"])
def test_one_token_reaches_what_follows_it(place, kind):
    """One mixer, one changed token: nothing before it moves, everything from it on does, across blocks, chunks and portions."""
    mix = {"memory": memory(2, 16, 16), "linear": linear(2, 16, 16, 0.999), "attention": attention(2, 1, 16, every=40, scale=0.05)}[kind]
    c = model([(mix, None)], vocab=50)
    w = weights_for(c, 3)
    w.update({k: v * 0 + (6.0 if k.endswith("f.b") else 0.0) for k, v in w.items() if k.endswith("f.b") or k.endswith("mix.f")})
    eng = InferenceEngine(EngineConfig(cache_type="none", max_batch_size=2, max_model_len=288, max_tokens_per_batch=288, num_kv_blocks=20,
                                       dtype=place[1], graph_batch_sizes=(1, 2)), config_from_dict(c), w, device=place[0])
    toks = tokens_for(c, 270, 9)
    for mark in (0, 15, 16, 127, 128, 200):
        other = list(toks)
        other[mark] = (toks[mark] + 7) % 50
        for portions in ([270], [3, 141] + [1] * 126, cut(270, 45)):
            x, y = feed_all(eng, toks, portions), feed_all(eng, other, portions)
            moved = (x - y).abs().amax(-1)
            assert (moved[:mark] == 0).all() and (moved[mark:] > 0).float().mean() > (0.98 if place[1] == "float32" else 0.8), (mark, portions)


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding(place):
    name = "mixed"
    toks = tokens_for(CONFIGS[name], 420, 31)
    agree(feed_all(engine(name, place), toks, [20] + [1] * 400), wanted(name, toks), place[1])


# ------------------------------------------------------------------------------------------ generation and scheduling
def check_greedy(name, prompt, sample, dtype):
    """fp32: the oracle's own greedy tokens. bf16: every chosen token is near the oracle's best, and its log-prob agrees."""
    w = {k: v.double() for k, v in weights_for(CONFIGS[name]).items()}
    ids = list(prompt) + list(sample.completion_tokens)
    lp = torch.log_softmax(oracle.forward(ids, w, CONFIGS[name])[len(prompt) - 1:-1], -1)
    tol = 5e-3 if dtype == "float32" else 2.5
    for row, tok, got in zip(lp, sample.completion_tokens, sample.logprobs):
        assert row[tok] > row.max() - tol and abs(row[tok] - got) < tol


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("cache,chunk", [("none", 0), ("radix", 13)])
def test_greedy_generation(place, cache, chunk):
    """A model with recurrent layers shares no prefixes, whatever cache is asked for."""
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
    w2 = weights_for(CONFIGS[name], seed=9)
    eng.update_weights(w2)
    want = oracle.forward(p[1], {k: v.double() for k, v in w2.items()}, CONFIGS[name])
    s = eng.open_stream()
    assert errors(eng.feed([(s, p[1], list(range(140)))]), want).median() < TOL[place[1]]


# ------------------------------------------------------------------------------------------ trace replay
def test_trace_replay_on_the_twins(tmp_path):
    name = "mixed"
    prompts = [tokens_for(CONFIGS[name], n, n) for n in (70, 30, 64)]
    save_safetensors_dir(weights_for(CONFIGS[name]), config_from_dict(CONFIGS[name]), tmp_path / "m")
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
    save_safetensors_dir(weights_for(CONFIGS[name]), config_from_dict(CONFIGS[name]), tmp_path / "m")
    lines, rows = trace_lines(prompts)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "112"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    by = dict(zip("abc", prompts))
    for i, want in enumerate(rows):
        e = errors(read_f32(tmp_path / f"{i}.f32", 97), torch.stack([wanted(name, by[k])[p_] for k, p_ in want]))
        assert e.median() < TOL[dtype]

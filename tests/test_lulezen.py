"""The Lulezen design in the framework against the plain oracle (``lulezen_oracle.py``): whole prompts, portions, decoding,
mixed batches, reused blocks, window edges, greedy generation through the scheduler, trace replay.

Every engine test runs on the CPU twins of the ops (fp32) and, on a GPU, in both number formats. Random weights are scaled so
that attention is peaked and every mechanism moves the logits; ``test_oracle_mistakes_show`` plants mistakes in the oracle
and checks that each is far outside the tolerances used here.
"""

import json
import math
import os
import subprocess
import sys

import lulezen_oracle as oracle
import pytest
import torch

from research_b200.inference import EngineConfig, InferenceEngine, SamplingParams
from research_b200.inference.trace_replay import make_engine, replay
from research_b200.models import config_from_dict, get_preset, init_random_weights, load_config, load_safetensors_dir, save_safetensors_dir
from research_b200.models.stack import LayerStackConfig

PLACES = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]
TOL = {"float32": 1e-5, "bfloat16": 0.07}      # worst row; rounding alone gives 3e-6 and (peaked scores) up to 0.05
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def mixer(heads=3, dim=24, rot=8, vdim=20, kv_rank=40, q_rank=36, window=20, base=1e4, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
        "rot": {"base": base, "dims": rot}, "scale": (dim + rot) ** -0.5 if scale is None else scale}}


def model(layers, vocab=130, width=56, cap=6.0, eps=1e-5):
    return {"architecture": "Lulezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": [{**m, "mlp": None if ff is None else {"kind": "dense", "ff": ff[0], "limit": ff[1]}} for m, ff in layers]}


CONFIGS = {
    "uneven": model([(mixer(), (72, 1.5)), (mixer(heads=5, dim=40, rot=16, vdim=12, kv_rank=24, q_rank=50, window=37, base=500.0, scale=0.3), None),
                     (mixer(window=1000), (100, 3.0))]),
    "one_head": model([(mixer(heads=1, dim=10, rot=4, vdim=9, kv_rank=11, q_rank=7, window=16), (17, 0.7)),
                       (mixer(heads=1, dim=10, rot=4, vdim=9, kv_rank=11, q_rank=7, window=1), (17, 0.7))], vocab=61, width=30, eps=1e-3),
    "wide_heads": model([(mixer(heads=2, dim=128, rot=64, vdim=128, kv_rank=160, q_rank=96, window=70), (256, 4.0)),
                         (mixer(heads=24, dim=16, rot=8, vdim=16, kv_rank=64, q_rank=48, window=33), (64, 1.0))], vocab=97, width=72, cap=9.0),
    "no_expand": model([(mixer(heads=2, dim=136, rot=72, vdim=40, kv_rank=300, q_rank=44, window=45), (40, 2.0))], vocab=83, width=48),
}


def weights_for(config, seed=0):
    """Random weights that make every part count: peaked scores, sinks of a few units, uneven norms, biases and scales. All
    values are exact in bf16, so that both number formats and the oracle see the same model."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in config_from_dict(config).param_shapes().items():
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last == "sink":
            t = 1.5 * r + 1.0
        elif last == "b":
            t = 0.5 * r
        elif len(shape) == 1:
            t = 1.0 + 0.3 * r
        else:
            gain = {"uq": 1.3, "uk": 1.3, "dkv": 1.0, "gate": 1.5, "up": 1.5, "head": 3.0, "embed": 1.0}.get(last, 1.0)
            t = r * gain / (math.sqrt(shape[1]) if name != "embed" else 1.0)
        out[name] = t.bfloat16()
    return out


def tokens_for(config, n, seed):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_CACHE = {}


def wanted(name, tokens):
    """Oracle logits in float64, remembered per prompt."""
    key = (name, tuple(tokens))
    if key not in _CACHE:
        w = {k: v.double() for k, v in weights_for(CONFIGS[name]).items()}
        _CACHE[key] = oracle.forward(tokens, w, CONFIGS[name])
    return _CACHE[key]


def error(got, want):
    """Largest rms difference of a row, relative to the spread of the expected logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()).max().item()


def engine(name, place, **kw):
    opts = dict(cache_type="none", max_batch_size=4, max_model_len=320, max_tokens_per_batch=400, num_kv_blocks=64, ignore_eos=True,
                dtype=place[1], graph_batch_sizes=(1, 2, 4))
    opts.update(kw)
    return InferenceEngine(EngineConfig(**opts), config_from_dict(CONFIGS[name]), weights_for(CONFIGS[name]), device=place[0])


def feed_all(eng, tokens, portions):
    """Logits of every position, fed in the given portions."""
    s, at, rows = eng.open_stream(), 0, []
    for n in portions:
        part = tokens[at:at + n]
        rows.append(eng.feed([(s, part, list(range(len(part))))]).cpu())
        at += n
    assert at >= len(tokens)
    eng.close_stream(s)
    return torch.cat(rows)


def cut(total, size):
    return [min(size, total - i) for i in range(0, total, size)]


# ------------------------------------------------------------------------------------------ configuration and weights
def test_config_round_trip_registry_and_checkpoint(tmp_path):
    for c in CONFIGS.values():
        cfg = config_from_dict(c)
        assert isinstance(cfg, LayerStackConfig) and config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    cfg = config_from_dict(CONFIGS["uneven"])
    assert [x.mlp is None for x in cfg.layers] == [False, True, False] and "l1.norm2" not in cfg.param_shapes()
    w = weights_for(CONFIGS["uneven"])
    save_safetensors_dir(w, cfg, tmp_path)
    assert load_config(tmp_path) == cfg
    back, cfg2 = load_safetensors_dir(tmp_path)
    assert cfg2 == cfg and all(torch.equal(back[k], v) for k, v in w.items())
    with pytest.raises(ValueError, match="unknown architecture"):
        config_from_dict({**CONFIGS["uneven"], "architecture": "Other"})
    bad = json.loads(json.dumps(CONFIGS["uneven"]))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        config_from_dict(bad)
    bad = json.loads(json.dumps(CONFIGS["uneven"]))
    bad["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        config_from_dict(bad)
    r = init_random_weights(get_preset("tiny-lulezen"), seed=3)
    assert r["l0.norm1"].eq(1).all() and r["l0.mix.sink"].eq(0).all() and r["final.norm.b"].eq(0).all() and r["l0.mix.o"].std() > 0
    assert get_preset("tiny-lulezen").num_params() == sum(t.numel() for t in r.values())


def test_oracle_mistakes_show(monkeypatch):
    """Each planted mistake moves some logits by far more than the tolerances of the engine tests."""
    c = CONFIGS["uneven"]
    w = {k: v.double() for k, v in weights_for(c).items()}
    toks = tokens_for(c, 60, 1)
    right = oracle.forward(toks, w, c)

    def wrong(change_config=None, change_weights=None):
        c2 = json.loads(json.dumps(c))
        w2 = dict(w)
        if change_config:
            change_config(c2)
        if change_weights:
            change_weights(w2)
        return error(oracle.forward(toks, w2, c2), right)

    def window(d):
        return lambda x: x["layers"][0]["mixer"]["mask"].update(size=20 + d)

    least = 1.5 * TOL["bfloat16"]
    assert wrong(window(1)) > least and wrong(window(-1)) > least
    assert wrong(None, lambda x: x.update({"l0.mix.sink": x["l0.mix.sink"] - 1e4})) > least
    assert wrong(None, lambda x: x.update({"l0.mix.g": x["l0.mix.g"] * 0})) > least
    assert wrong(None, lambda x: x.update({"l2.norm2.b": x["l2.norm2.b"] * 0})) > least
    assert wrong(None, lambda x: x.update({"l1.ls1": torch.ones_like(x["l1.ls1"])})) > least
    assert wrong(lambda x: x["layers"][0]["mlp"].update(limit=1e9)) > least
    assert wrong(lambda x: x["layers"][1]["mixer"]["rot"].update(base=600.0)) > TOL["bfloat16"]
    assert wrong(lambda x: x.update(logit_softcap=1e9)) > TOL["bfloat16"]
    monkeypatch.setattr(oracle, "rotate", lambda v, *_: v)
    assert error(oracle.forward(toks, w, c), right) > least


# ------------------------------------------------------------------------------------------ logits through the engine
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_portions_and_single_tokens(name, place):
    toks = tokens_for(CONFIGS[name], 150, 5)
    want = wanted(name, toks)
    eng = engine(name, place)
    for portions in ([150], cut(150, 17), cut(150, 2), [1, 48, 3, 16, 2, 80], [5] + [1] * 30 + [40] + [1] * 75):
        assert error(feed_all(eng, toks, portions), want) < TOL[place[1]], portions
    assert eng.check_invariants() == 0 and eng.cache_stats()["free_blocks"] == 64
    if place == ("cuda", "bfloat16"):
        assert eng.runner.layers[0].mixer.expand == (name != "no_expand")


@pytest.mark.parametrize("place", PLACES)
def test_unequal_requests_in_one_batch_and_reused_blocks(place):
    """Portions beside single tokens, requests that pause, a pool that only fits the live ones: rows equal the request alone."""
    name = "uneven"
    prompts = {k: tokens_for(CONFIGS[name], n, 20 + i) for i, (k, n) in enumerate({"a": 90, "b": 40, "c": 1, "d": 70, "e": 60, "f": 90}.items())}
    eng = engine(name, place, num_kv_blocks=20)            # a + b + d are 6 + 3 + 5 blocks; all six would need 25
    steps = [{"a": 30, "b": 2, "c": 1}, {"a": 1, "b": 20, "d": 33}, {"a": 1, "d": 2}, {"a": 20, "b": 1, "d": 1}, {"b": 17, "a": 2},
             {"a": 36, "d": 34}, {"e": 3, "f": 50}, {"e": 1, "f": 1}, {"f": 39, "e": 56}]
    at, streams = dict.fromkeys(prompts, 0), {}
    for step in steps:
        entries, order = [], []
        for k, n in step.items():
            streams.setdefault(k, None)
            if streams[k] is None:
                streams[k] = eng.open_stream()
            entries.append((streams[k], prompts[k][at[k]:at[k] + n], list(range(n))))
            order += [(k, p) for p in range(at[k], at[k] + n)]
            at[k] += n
        got = eng.feed(entries)
        want = torch.stack([wanted(name, prompts[k])[p] for k, p in order])
        assert error(got, want) < TOL[place[1]], step
        for k in step:
            if at[k] == len(prompts[k]):
                eng.close_stream(streams[k])
    assert all(at[k] == len(p) for k, p in prompts.items())
    assert eng.cache_stats()["free_blocks"] == 20 and eng.check_invariants() == 0
    s = eng.open_stream()
    with pytest.raises(RuntimeError, match="full"):
        eng.feed([(s, [1] * 318, []), (eng.open_stream(), [1] * 40, [])])
    assert eng.cache_stats()["free_blocks"] == 20          # nothing was taken by the refused step
    assert eng.feed([(s, [1, 2, 3], [])]) is None
    with pytest.raises(RuntimeError, match="unknown stream"):
        eng.feed([(10**6, [1], [])])


@pytest.mark.parametrize("place", PLACES)
def test_window_edges_in_prompts_and_decoding(place):
    """One layer, one marked token far back: changing it must reach exactly the positions whose window holds it."""
    c = model([(mixer(window=18), None)], vocab=50)
    w = weights_for(c, 3)
    eng = InferenceEngine(EngineConfig(cache_type="none", max_batch_size=2, max_model_len=128, max_tokens_per_batch=128, num_kv_blocks=16,
                                       dtype=place[1], graph_batch_sizes=(1, 2)), config_from_dict(c), w, device=place[0])
    toks = tokens_for(c, 100, 9)
    for mark in (0, 15, 16, 31, 40):
        other = list(toks)
        other[mark] = (toks[mark] + 7) % 50
        for portions in ([100], [3, 41] + [1] * 56, cut(100, 19)):
            a, b = feed_all(eng, toks, portions), feed_all(eng, other, portions)
            moved = (a - b).abs().amax(-1)
            seen = torch.arange(100)
            seen = (seen >= mark) & (seen < mark + 18)
            assert (moved[seen] > 0).all() and (moved[~seen] == 0).all(), (mark, portions)


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding(place):
    name = "uneven"
    toks = tokens_for(CONFIGS[name], 300, 31)
    got = feed_all(engine(name, place), toks, [20] + [1] * 280)
    assert error(got, wanted(name, toks)) < TOL[place[1]]


# ------------------------------------------------------------------------------------------ generation and scheduling
def check_greedy(name, prompt, sample, dtype):
    """fp32: the oracle's own greedy tokens. bf16: every chosen token is near the oracle's best, and its log-prob agrees."""
    w = {k: v.double() for k, v in weights_for(CONFIGS[name]).items()}
    ids = list(prompt) + list(sample.completion_tokens)
    lp = torch.log_softmax(oracle.forward(ids, w, CONFIGS[name])[len(prompt) - 1:-1], -1)
    tol = 1e-3 if dtype == "float32" else 0.6
    for row, tok, got in zip(lp, sample.completion_tokens, sample.logprobs):
        assert row[tok] > row.max() - tol and abs(row[tok] - got) < tol


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("cache,chunk", [("none", 0), ("none", 11), ("radix", 0), ("radix", 13), ("paged", 13)])
def test_greedy_generation(place, cache, chunk):
    name = "uneven"
    shared = tokens_for(CONFIGS[name], 40, 50)
    prompts = [shared + tokens_for(CONFIGS[name], n, 60 + n) for n in (3, 30, 17)] + [tokens_for(CONFIGS[name], n, 80 + n) for n in (1, 2, 60)]
    eng = engine(name, place, cache_type=cache, prefill_chunk=chunk, num_kv_blocks=80)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9))
    for p, s in zip(prompts, outs):
        assert s.prompt_tokens == tuple(p) and len(s.completion_tokens) == 9
        check_greedy(name, p, s, place[1])
    again = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9))
    for p, s in zip(prompts, again):
        check_greedy(name, p, s, place[1])
    if cache != "none":
        assert eng.cache_stats()["hit_tokens"] > 0 and max(s.cached_tokens for s in again) >= 32
    assert eng.check_invariants() == 0 and not eng.has_pending()


@pytest.mark.parametrize("place", PLACES)
def test_prompt_longer_than_a_step_and_preemption(place):
    """A prompt beyond the step's token budget goes in portions beside decoding rows; a pool too small for all preempts."""
    name = "uneven"
    prompts = [tokens_for(CONFIGS[name], n, 90 + n) for n in (150, 20, 33, 75)]
    eng = engine(name, place, max_tokens_per_batch=40, num_kv_blocks=17)
    joint = []
    step = eng._step_with_ids

    def watch():
        r = step()
        joint.append(eng.last_step_rows)
        return r

    eng._step_with_ids = watch
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=25))
    for p, s in zip(prompts, outs):
        assert len(s.completion_tokens) == 25
        check_greedy(name, p, s, place[1])
    assert any(a and b for a, b in joint), "no step mixed portions with decoding rows"
    assert eng.check_invariants() == 0 and eng.cache_stats()["free_blocks"] == 17


def test_portions_respect_the_step_budget():
    name = "one_head"
    eng = engine(name, ("cpu", "float32"), max_tokens_per_batch=24, prefill_chunk=10)
    seen = []
    build = eng._build_packed

    def watch(which, rows):
        out = build(which, rows)
        seen.append(out[1:3])
        return out

    eng._build_packed = watch
    eng.generate([tokens_for(CONFIGS[name], n, n) for n in (50, 31, 12, 3)], SamplingParams(temperature=0.0, max_tokens=6))
    assert seen and all(total <= 24 and longest <= 10 for total, longest in seen)


@pytest.mark.parametrize("place", PLACES)
def test_seeded_sampling_weight_update_and_score(place):
    name = "uneven"
    eng = engine(name, place, cache_type="radix", num_kv_blocks=80)
    p = [tokens_for(CONFIGS[name], 25, 1), tokens_for(CONFIGS[name], 40, 2)]
    a = eng.generate(p, SamplingParams(temperature=1.0, max_tokens=6, seed=7))
    b = eng.generate(p, SamplingParams(temperature=1.0, max_tokens=6, seed=7))
    assert [s.completion_tokens for s in a] == [s.completion_tokens for s in b]
    assert error(eng.runner.score(torch.tensor(p[1])), wanted(name, p[1])) < TOL[place[1]]
    w2 = weights_for(CONFIGS[name], seed=9)
    eng.update_weights(w2)
    want = oracle.forward(p[0], {k: v.double() for k, v in w2.items()}, CONFIGS[name])
    s = eng.open_stream()
    assert error(eng.feed([(s, p[0], list(range(25)))]), want) < TOL[place[1]]
    assert eng.generate(p[:1], SamplingParams(temperature=0.0, max_tokens=2))[0].cached_tokens == 0


def test_http_front_end_serves_it():
    from fastapi.testclient import TestClient

    from research_b200.inference.server import EngineService, create_app

    name = "uneven"
    svc = EngineService(engine(name, ("cpu", "float32"), cache_type="radix", num_kv_blocks=80))
    try:
        client = TestClient(create_app(svc, name))
        ids = tokens_for(CONFIGS[name], 30, 4)
        r = client.post("/generate", json={"input_ids": ids, "sampling_params": {"temperature": 0.0, "max_new_tokens": 5}}).json()
        w = {k: v.double() for k, v in weights_for(CONFIGS[name]).items()}
        for k, tok in enumerate(r["output_ids"]):
            assert int(oracle.forward(ids + r["output_ids"][:k], w, CONFIGS[name])[-1].argmax()) == tok
    finally:
        svc.shutdown()


def test_sizes_beyond_the_kernels_are_refused():
    c = model([(mixer(kv_rank=1500), None)])
    with pytest.raises(ValueError, match="latent channels"):
        InferenceEngine(EngineConfig(max_batch_size=2, max_model_len=64, num_kv_blocks=8), config_from_dict(c), weights_for(c), device="cpu")


def test_hf_models_take_portions_and_fed_tokens_too():
    """The portioned scheduler and fed streams are not special to layer stacks."""
    from research_b200.models import causal_lm_forward

    cfg = get_preset("tiny-qwen2", num_layers=2)
    w = init_random_weights(cfg, seed=0)
    toks = torch.randint(0, cfg.vocab_size, (70,), generator=torch.Generator().manual_seed(1)).tolist()
    want = causal_lm_forward(torch.tensor([toks]), w, cfg)[0]
    res = []
    for chunk in (0, 16):
        eng = InferenceEngine(EngineConfig(cache_type="radix", max_batch_size=4, max_model_len=128, num_kv_blocks=40, ignore_eos=True,
                                           prefill_chunk=chunk), cfg, w, device="cpu")
        res.append([s.completion_tokens for s in eng.generate([toks, toks[:33], toks[:5]], SamplingParams(temperature=0.0, max_tokens=5))])
        got = feed_all(eng, toks, [30, 1, 2, 20] + [1] * 17)
        assert (got - want).abs().max() < 1e-3 and eng.check_invariants() == 0
    assert res[0] == res[1]


# ------------------------------------------------------------------------------------------ trace replay
def trace_lines(prompts):
    """Two interleaved requests and one that reuses the first one's blocks."""
    a, b, c = prompts
    steps = [([("a", a[:40], [0, 39]), ("b", b[:3], [])], []), ([("a", a[40:], [0]), ("b", b[3:4], [0])], ["a"]),
             ([("b", b[4:], [1, len(b) - 5])], ["b"]), ([("c", c, [len(c) - 1, 2])], ["c"])]
    rows = [[("a", 0), ("a", 39)], [("a", 40), ("b", 3)], [("b", 5), ("b", len(b) - 1)], [("c", len(c) - 1), ("c", 2)]]
    return [json.dumps({"step": i, "entries": [{"id": k, "tokens": t, "want": w} for k, t, w in e], "end": end}) for i, (e, end) in enumerate(steps)], rows


def read_f32(path, vocab):
    return torch.frombuffer(bytearray(path.read_bytes()), dtype=torch.float32).view(-1, vocab)


def test_trace_replay_on_the_twins(tmp_path):
    name = "uneven"
    prompts = [tokens_for(CONFIGS[name], n, n) for n in (70, 30, 64)]
    save_safetensors_dir(weights_for(CONFIGS[name]), config_from_dict(CONFIGS[name]), tmp_path / "m")
    eng = make_engine(str(tmp_path / "m"), "float32", 112, device="cpu")
    lines, rows = trace_lines(prompts)
    done = []
    replay(eng, lines, tmp_path, done.append)
    by = dict(zip("abc", prompts))
    for i, want in enumerate(rows):
        got = read_f32(tmp_path / f"{i}.f32", 130)
        assert error(got, torch.stack([wanted(name, by[k])[p] for k, p in want])) < TOL["float32"]
    assert done == [0, 1, 2, 3] and eng.cache_stats()["free_blocks"] == 7


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(tmp_path, dtype, cuda_device):
    name = "wide_heads"
    prompts = [tokens_for(CONFIGS[name], n, n) for n in (70, 30, 64)]
    save_safetensors_dir(weights_for(CONFIGS[name]), config_from_dict(CONFIGS[name]), tmp_path / "m")
    lines, rows = trace_lines(prompts)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "112"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    by = dict(zip("abc", prompts))
    for i, want in enumerate(rows):
        got = read_f32(tmp_path / f"{i}.f32", 97)
        assert error(got, torch.stack([wanted(name, by[k])[p_] for k, p_ in want])) < TOL[dtype]


def test_trace_run_refuses_a_model_without_a_32_bit_mode(tmp_path):
    get_preset("tiny-qwen2").save(tmp_path)
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "64"], input="", capture_output=True, text=True, timeout=300)
    assert p.returncode == 3

"""Replay of token traces: feed given tokens through the engine step by step and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N        (or: research-b200 replay ...)

Steps are read from standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one engine batch (``InferenceEngine.feed``): portions of prompts beside single tokens, from
the cache that earlier steps left. ``want`` names places among an entry's tokens; a step that wants something writes
``<out>/<step>.f32``, little-endian fp32 ``[wanted, vocab]`` in the order of the entries and of their places. ``end`` lists
the requests that give their cache blocks back after the step. Every step is answered with a line ``done <step>``.

``--max-tokens`` sizes the cache: tokens held by live requests at any time, each request rounded up to whole blocks.
At most four requests are live. Missing native libraries of the model are compiled first. Exit code 3: the model's
runner has no 32-bit mode.
"""

from __future__ import annotations

import argparse
import json
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

import torch

from .. import _native
from ..models.registry import architecture_of, load_config, runner_class
from .engine import InferenceEngine
from .model_runner import BLOCK
from .types import EngineConfig

MAX_LIVE = 4


def build_libraries(names: tuple[str, ...]) -> None:
    with ThreadPoolExecutor(max_workers=len(names)) as pool:
        list(pool.map(_native.build_one, names))


def make_engine(model: str, dtype: str, max_tokens: int, device: str | None = None) -> InferenceEngine:
    """An engine whose cache holds ``max_tokens`` and that keeps nothing of finished requests."""
    blocks = -(-max_tokens // BLOCK)
    tokens = blocks * BLOCK
    return InferenceEngine(EngineConfig(model_path=model, cache_type="none", max_batch_size=MAX_LIVE, max_model_len=tokens,
                                        max_tokens_per_batch=tokens, num_kv_blocks=blocks, dtype=dtype,
                                        graph_batch_sizes=tuple(range(1, MAX_LIVE + 1))), device=device)


def replay(engine: InferenceEngine, lines, out: Path, answer) -> None:
    """Run the steps in ``lines``; ``answer(step)`` after each one."""
    streams: dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in streams:
                streams[e["id"]] = engine.open_stream()
            entries.append((streams[e["id"]], e["tokens"], e["want"]))
        logits = engine.feed(entries) if entries else None
        if logits is not None:
            (out / f"{step['step']}.f32").write_bytes(logits.float().cpu().numpy().astype("<f4", copy=False).tobytes())
        engine.check_kernels()
        for name in step["end"]:
            engine.close_stream(streams.pop(name))
        answer(step["step"])


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given tokens through a model, step by step, and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    cfg = load_config(args.model)
    if args.dtype == "float32" and not runner_class(cfg).supports_f32:
        print("this model has no 32-bit mode", file=sys.stderr)
        return 3
    if not torch.cuda.is_available():
        print("a CUDA device is needed", file=sys.stderr)
        return 1
    build_libraries(architecture_of(json.loads((Path(args.model) / "config.json").read_text())).libraries)
    engine = make_engine(args.model, args.dtype, args.max_tokens, "cuda:0")
    replay(engine, sys.stdin, Path(args.out), lambda step: print(f"done {step}", flush=True))
    engine.shutdown()
    return 0


"""Which configuration class reads a ``config.json`` and which runner executes the model.

Hugging Face style files (``model_type`` / ``architectures``) are ``ModelConfig`` models run by ``ModelRunner``; files
that name an ``architecture`` listed here are layer stacks run by ``StackRunner``.
"""

from __future__ import annotations

import importlib
import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

from .config import ModelConfig
from .stack import LayerStackConfig


@dataclass(frozen=True)
class Architecture:
    parse: Callable[[dict], object]
    runner: str                        # module:class, imported when an engine is built
    libraries: tuple[str, ...]         # native libraries its kernels live in (names of ``_native.LIBRARIES``)


HF_DECODER = Architecture(ModelConfig.from_hf_dict, "research_b200.inference.model_runner:ModelRunner",
                          ("rb_engine_core", "rb_gemm", "rb_gemm2", "rb_ops", "rb_attn", "rb_flash", "rb_moe"))
ARCHITECTURES: dict[str, Architecture] = {
    "Lulezen": Architecture(LayerStackConfig.from_dict, "research_b200.inference.stack_runner:StackRunner",
                            ("rb_engine_core", "rb_gemm", "rb_gemm2", "rb_gemm_f32", "rb_ops", "rb_latent", "rb_flash")),
    "Zamusun": Architecture(LayerStackConfig.from_dict, "research_b200.inference.stack_runner:StackRunner",
                            ("rb_engine_core", "rb_gemm", "rb_gemm2", "rb_gemm_f32", "rb_ops", "rb_recurrent", "rb_attn", "rb_flash", "rb_moe")),
    "Sumitar": Architecture(LayerStackConfig.from_dict, "research_b200.inference.stack_runner:StackRunner",
                            ("rb_engine_core", "rb_gemm", "rb_gemm2", "rb_gemm_f32", "rb_ops", "rb_recurrent", "rb_attn", "rb_flash", "rb_moe")),
    "Fogurax": Architecture(LayerStackConfig.from_dict, "research_b200.inference.stack_runner:StackRunner",
                            ("rb_engine_core", "rb_gemm", "rb_gemm2", "rb_gemm_f32", "rb_ops", "rb_recurrent", "rb_attn", "rb_flash", "rb_moe")),
}


def architecture_of(d: dict) -> Architecture:
    name = d.get("architecture")
    if name is None:
        return HF_DECODER
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)} and the Hugging Face families")
    return ARCHITECTURES[name]


def config_from_dict(d: dict):
    return architecture_of(d).parse(d)


def load_config(path: str | Path):
    """The model configuration in ``path/config.json``."""
    return config_from_dict(json.loads((Path(path) / "config.json").read_text()))


def runner_class(cfg):
    arch = ARCHITECTURES[cfg.architecture] if isinstance(cfg, LayerStackConfig) else HF_DECODER
    module, _, name = arch.runner.partition(":")
    return getattr(importlib.import_module(module), name)

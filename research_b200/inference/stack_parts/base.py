"""What parts of a layer stack have in common."""

from __future__ import annotations

import weakref
from typing import Any, Callable

import torch

Getter = Callable[[str], torch.Tensor]       # checkpoint tensor by name, on the runner's device


def up(n: int, m: int) -> int:
    return -(-n // m) * m


class Part:
    """A kind of mixer or feed-forward in one runner. ``forward`` reads the activations ``inp [T, wp]`` and, for mixers and dense
    feed-forwards, fills ``y [T, wp]`` (fp32)."""

    # mixers: the layer's narrow fp32 projection rides along as the last rows of the mixer's joint projection (``make`` is told how
    # many) and ``project`` fills it; otherwise the runner multiplies it on its own
    fuses_tail = False

    def __init__(self, runner):
        self.r = weakref.proxy(runner)       # no cycle: the runner's graphs go when its engine does
        self.layers: list[Any] = []          # weights made so far
        self._planned: tuple = (None, None)
        self.specs: list[Any] = []

    # ---- sizing, before a runner exists
    @staticmethod
    def cache_row_elements(spec) -> int:
        """Cached elements per token and layer run."""
        return 0

    @staticmethod
    def state_floats(spec) -> int:
        """fp32 elements of recurrent state per sequence and layer run."""
        return 0

    @staticmethod
    def small_rows(spec) -> int:
        """Rows of the layer's narrow projection with fp32 results (gate logits, router)."""
        return 0

    # ---- memory
    def zeros(self, *shape: int, dtype: torch.dtype | None = None) -> torch.Tensor:
        return torch.zeros(*shape, dtype=dtype or self.r.dtype, device=self.r.device)

    def make(self, spec, tail: int = 0):
        raise NotImplementedError

    def new_cache(self, w):
        return None

    def allocate(self) -> None:
        pass

    # ---- weights
    def load(self, w, get: Getter, p: str) -> None:
        raise NotImplementedError

    def load_small(self, w, get: Getter, p: str, dst: torch.Tensor) -> None:
        pass

    # ---- one step
    def plan(self, b) -> Any:
        return None

    def planned(self, b) -> Any:
        """``plan(b)``, made once per batch (a part may also belong to another one)."""
        if self._planned[0] is not b:
            self._planned = (b, self.plan(b))
        return self._planned[1]

    def project(self, w, inp: torch.Tensor, tail: torch.Tensor | None) -> None:
        """First half of a mixer: its projections of ``inp``, and the narrow one into ``tail`` (fp32)."""


def load_heads(dst: torch.Tensor, src: torch.Tensor, heads: int, dim: int, padded: int) -> None:
    """``src [heads*dim, d]`` into the leading rows of every head's block of ``dst [heads*padded, >= d]``."""
    dst.unflatten(0, (heads, padded))[:, :dim, :src.shape[1]].copy_(src.view(heads, dim, -1))


def load_head_vector(dst: torch.Tensor, src: torch.Tensor, heads: int, dim: int, padded: int) -> None:
    dst.view(heads, padded)[:, :dim].copy_(src.view(heads, dim))


def load_head_columns(dst: torch.Tensor, src: torch.Tensor, heads: int, dim: int, padded: int) -> None:
    """``src [d, heads*dim]`` into the leading columns of every head's block of ``dst [>= d, heads*padded]``."""
    d = src.shape[0]
    dst[:d].unflatten(1, (heads, padded))[:, :, :dim].copy_(src.view(d, heads, dim))

"""What every part of a layer has in common, the registries of part kinds, and what a
mixer may ask of the cache manager.

A part is built from a :class:`~rllm_b200.config.base.PartSpec` (its kind, its sizes and
constants, the prefix of its tensors) and a :class:`Runtime`.  It says which tensors it
expects (`expected_tensors`), takes them (`load`), and is then called by its block.  No part
knows which model it is in.  A new kind is added with ``@register_part(category, kind)``:
nothing else in the package has to change.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Mapping, Optional

import torch

CATEGORIES = ("embedding", "norm", "position", "mixer", "ffn", "block", "lm_head", "junction", "side")
_REGISTRY: dict[str, dict[str, Callable]] = {c: {} for c in CATEGORIES}


class PartError(ValueError):
    pass


def register_part(category: str, kind: str):
    """Class decorator: makes `kind` available in `category` ('mixer', 'ffn', 'norm', ...)."""
    if category not in _REGISTRY:
        raise PartError(f"unknown part category {category!r} (known: {', '.join(CATEGORIES)})")

    def deco(cls):
        _REGISTRY[category][kind] = cls
        return cls
    return deco


def part_class(category: str, kind: str):
    try:
        return _REGISTRY[category][kind]
    except KeyError:
        raise PartError(f"no {category} part of kind {kind!r} is registered "
                        f"(registered: {', '.join(sorted(_REGISTRY.get(category, {})))})") from None


def build_part(category: str, spec, runtime: "Runtime", **extra):
    return part_class(category, spec.kind)(dict(spec.params), spec.prefix, runtime, **extra)


@dataclass(frozen=True)
class Runtime:
    """Where and in which precision a model runs.  `dtype` is the storage type of weights,
    activations between kernels and the cache (bfloat16 or float32); the residual stream,
    norms' statistics, softmax, rotation angles and logits are float32 in both."""
    device: torch.device
    dtype: torch.dtype

    @property
    def is_f32(self) -> bool:
        return self.dtype == torch.float32


# ---------------------------------------------------------------- what a mixer asks of the cache

@dataclass(frozen=True)
class PagedKVNeed:
    """Keys and values in pages.  `window` > 0: only the last `window` keys are ever read, so
    pages that the window has passed can be given back; with `keep_first` > 0 the first that many
    keys of a request stay readable all the same, and their pages are kept.  `v_head_dim`: size of
    a value head where it differs from a key head (0: the same).  `values_in_keys` > 0: the values
    are the first that many entries of the key rows themselves (attention through a latent that
    serves as key and value); there is no pool of values then, and a view's `v` is its `k`."""
    num_kv_heads: int
    head_dim: int
    window: int = 0
    keep_first: int = 0
    v_head_dim: int = 0
    values_in_keys: int = 0

    @property
    def value_dim(self) -> int:
        return self.v_head_dim or self.head_dim


@dataclass(frozen=True)
class StateNeed:
    """A fixed-size state per request (any shape), kept in a slot for the request's lifetime
    and zeroed when the slot is taken."""
    shape: tuple
    dtype: torch.dtype = torch.float32


class Part:
    """Base of all parts."""

    # True for a part whose `forward` may be captured into a CUDA graph and replayed for another step
    # of the same padded shape: it launches kernels and torch operations on device tensors only, reads
    # nothing back to the host, and takes from the step's host copies (`ctx.q_lens`, `ctx.start_pos`,
    # ...) no more than the shape.  Padding rows of such a step have slot -1 in the pages and the last
    # state slot, which belongs to no request.  A model with a part that does not say so runs eagerly.
    CAPTURE_SAFE = False

    # True for a part that touches device memory through the launchers of csrc/ops only (no torch
    # operation of its own on tensors): the launches of a layer of such parts can be recorded once and
    # replayed for the other layers of the same build (models/model.py, ops.Trace).
    TRACEABLE = False

    def __init__(self, params: Mapping[str, Any], prefix: str, runtime: Runtime):
        self.params = dict(params)
        self.prefix = prefix
        self.runtime = runtime

    def expected_tensors(self) -> dict:
        """Full tensor name -> (shape, role); role 'norm' marks weights that start at 1."""
        return {}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        """Takes the tensors named by `expected_tensors` (CPU, as stored) and keeps device copies."""

    def _to_device(self, t: torch.Tensor, dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        return t.to(device=self.runtime.device, dtype=dtype or self.runtime.dtype).contiguous()


class Mixer(Part):
    """Token mixer interface.

    ``cache_need()`` returns a PagedKVNeed, a StateNeed, None, or a tuple of needs (a mixer that is
    several mixers side by side); `cache` is then a tuple of views in the same order.
    ``forward(h, ctx, cache, position)``: `h` [n, hidden] normed activations in the runtime's
    dtype, `ctx` the step's :class:`~rllm_b200.engine.batch.StepContext`, `cache` the view of
    this run entry's cache (:class:`~rllm_b200.cache.views.PagedKVView` or ``StateView``; None
    if it needs none), `position` the layer's position-encoding part or None, `residual` the
    float32 residual stream [n, hidden].  Returns the mixer's output [n, hidden] (float32 or the
    runtime's dtype), which the block adds to the residual stream; or adds it into `residual`
    itself and returns None."""

    def cache_need(self):
        return None

    def forward(self, h, ctx, cache, position, residual=None):
        raise NotImplementedError


class FeedForward(Part):
    """``forward(h, ctx, residual=None)`` -> [n, hidden] or None.  As for mixers, a part may add
    its output into the float32 `residual` itself and return None."""

    def forward(self, h, ctx, residual=None):
        raise NotImplementedError


class Norm(Part):
    """``forward(x, delta=None, rows=None, write_x=True, delta_scale=1.0)``: adds `delta_scale *
    delta` to the float32 residual stream `x` (in place when write_x), optionally gathers `rows`,
    returns the normed rows in the runtime's dtype."""

    def forward(self, x, delta=None, rows=None, write_x=True, delta_scale=1.0):
        raise NotImplementedError


class Side(Part):
    """A part that joins something of its own to the stream behind a layer's sublayers:
    ``forward(x, rows, ctx, mult, next_norm=None)``: x += mult * (what the part makes of `rows`), with `x`
    the float32 stream and `rows` the same rows as a product's operand (the runtime's type).  With
    `next_norm` (the norm that reads the stream next) the part may make that norm's rows in the kernel
    that joins, and returns them; else None."""

    def forward(self, x, rows, ctx, mult, next_norm=None):
        raise NotImplementedError


class Junction(Part):
    """A part that stands between two run entries and rewrites the whole residual stream:
    ``forward(x, x0, delta, delta_scale, arg) -> new x`` with `x` the float32 stream, `delta` what
    the block before still owes it (or None), `x0` the embedding output of the step's tokens and
    `arg` the run entry's `junction_arg`."""

    def forward(self, x, x0, delta, delta_scale, arg):
        raise NotImplementedError

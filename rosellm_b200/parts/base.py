"""Interfaces of the parts a model is assembled from, and their registry.

A part is constructed from its ``PartSpec.params`` alone: sizes, constants and
options.  It declares the tensors it needs (``param_specs``), what cache or
per-request state it wants (``cache_spec`` / ``state_spec``), receives its
tensors with ``bind`` and does its work on one step's tokens in ``forward``.
No part knows which model it is in.

Categories and the signature of ``forward``:

``embedding``      ``forward(ctx, position) -> x``: the residual stream
                   ``[tokens, hidden]`` in float32 for ``ctx.token_ids``.
``position``       ``table()``: a learned table the embedding adds, or ``None``;
                   ``rotate(ctx, q, k)``: in-place encoding of queries and keys.
``norm``           ``forward(ctx, x, rows=None) -> h``: normalised rows of the
                   residual stream in the activation dtype.
``mixer``          ``forward(ctx, run, h, x, add=True)``: mixes tokens of a request and
                   adds the result to ``x`` in place (``add=False``: writes it
                   there instead, for blocks that normalise a sublayer's output
                   before it joins the stream).  ``run`` tells which layer's
                   cache or state to use and whether to append to it.
``feed_forward``   ``forward(ctx, h, x, add=True)``: adds its result to ``x`` in
                   place, or with ``add=False`` writes it there.
``block``          ``forward(ctx, run, layer, x)``: arranges norms, mixer and
                   feed-forward of one layer around the residual stream.
``head``           ``forward(ctx, h) -> logits`` ``[rows, vocab]`` float32.
``stream_input``   ``forward(ctx, x, first=False, layer=None, **args)``: adds something to the stream between
                   two runs of layers (``ModelSpec.stream_inputs`` says where and with which ``args``;
                   ``first``: the stream is the embedding's output as it stands; ``layer``: the layer that
                   runs next, given to the last input ahead of it, which may leave that layer's first norm
                   in ``ctx.extras["normed_ahead"]`` if the layer's block says it takes it);
                   ``keep_embedding(ctx, x)`` is called right after the embedding for a part none of whose
                   inputs comes first.
``connection``     how a sublayer reads and writes a stream of another form than one row a token (weights that a
                   block arranging such a stream uses: ``parts/hyper.py``).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Callable

import torch

CATEGORIES = ("embedding", "position", "norm", "mixer", "feed_forward", "block", "head", "stream_input", "connection")

_PARTS: dict[tuple[str, str], type] = {}


def register_part(category: str, kind: str) -> Callable[[type], type]:
    """Class decorator: make ``kind`` constructible for ``category``."""
    if category not in CATEGORIES:
        raise ValueError(f"unknown part category {category!r}; one of {CATEGORIES}")

    def deco(cls: type) -> type:
        _PARTS[(category, kind)] = cls
        cls.category = category
        cls.kind = kind
        return cls

    return deco


def unregister_part(category: str, kind: str) -> None:
    _PARTS.pop((category, kind), None)


def part_class(category: str, kind: str) -> type:
    try:
        return _PARTS[(category, kind)]
    except KeyError:
        known = sorted(k for c, k in _PARTS if c == category)
        raise KeyError(f"no {category} part named {kind!r}; registered: {known}") from None


@dataclass(frozen=True)
class ParamSpec:
    """One tensor a part reads.

    ``role`` is the part's own name for it; the ``PartSpec.tensors`` map gives
    its name in the weight file.  ``shape`` is the shape in the file; an extent of -1 there is
    whatever the file has (a low rank that no configuration key gives: the part reads it off the
    tensor when it is bound; the random-weights mode needs it given).
    ``kind`` decides how it is kept on the device:
    ``matrix``: the engine's compute dtype (bfloat16 or float32);
    ``vector``: float32 in both modes (norm scales, biases: small, and read
    by 32-bit arithmetic); ``int_table``: int32.
    ``transpose``: the file holds ``[in, out]`` and the part wants ``[out, in]``.
    """

    role: str
    shape: tuple[int, ...]
    kind: str = "matrix"
    transpose: bool = False
    # how the random-weights mode fills it: "normal", "ones" (a norm's scale), "zeros" or "eye" (a square mixing matrix)
    init: str = "normal"
    # an integer table's entries lie in [0, below); the random-weights mode draws every row's entries distinct
    below: int = 0


@dataclass(frozen=True)
class KVCacheSpec:
    """Keys and values in pages.  ``window``: how many latest keys a query sees
    (``None``: all of them); older pages are given back while the request lives.
    ``chunks``: sizes of chunks, counted from the sequence's first token, of which a query sees its own alone.
    A spec with a window and chunks, or with chunks of several sizes, is that of a cache read by several layers: a
    page is kept while any of them sees into it (``covering``).
    ``planes``: 2 for keys and values kept apart; 1 where one cached row per token serves as
    both (a latent that the mixer's queries and outputs are projected onto)."""

    num_kv_heads: int
    head_dim: int
    window: int | None = None
    planes: int = 2
    chunks: tuple[int, ...] = ()

    @property
    def bounded(self) -> bool:
        """Whether keys are ever out of every later query's sight while the request lives."""
        return self.window is not None or bool(self.chunks)

    @property
    def reach(self) -> int:
        """The most keys a query sees (of a bounded spec)."""
        return max((self.window or 0, *self.chunks))

    def first_key(self, pos: int) -> int:
        """The earliest key that a query at ``pos`` or later sees."""
        if not self.bounded:
            return 0
        first = [pos // c * c for c in self.chunks]
        if self.window is not None:
            first.append(pos - self.window + 1)
        return max(0, min(first))

    def same_rows(self, other: "KVCacheSpec") -> bool:
        """Whether both describe the same cached rows, whatever of them is in sight."""
        return (self.num_kv_heads, self.head_dim, self.planes) == (other.num_kv_heads, other.head_dim, other.planes)

    def covering(self, other: "KVCacheSpec") -> "KVCacheSpec":
        """The same rows, kept for this spec's queries and the other's."""
        if not (self.bounded and other.bounded):
            return replace(self, window=None, chunks=())
        windows = [w for w in (self.window, other.window) if w is not None]
        return replace(self, window=max(windows, default=None), chunks=tuple(sorted(set(self.chunks) | set(other.chunks))))


@dataclass(frozen=True)
class StateSpec:
    """Per-request state of fixed size, one slot per live request."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


class Part:
    category = ""
    kind = ""

    def param_specs(self) -> list[ParamSpec]:
        return []

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        """Receive the device tensors named by ``param_specs`` (by role)."""
        for role, t in tensors.items():
            setattr(self, role, t)

    def cache_spec(self) -> KVCacheSpec | None:
        return None

    def state_spec(self) -> StateSpec | None:
        return None

    # whether ``forward`` may be captured in a CUDA graph (no host reads,
    # no allocation whose address changes between replays)
    graph_safe = False

    # whether ``forward`` does all its device work through ``rosellm_b200.ops.kernels`` (no torch
    # operation on device tensors) and chooses it from the step's sizes and ``launch_key`` alone
    launches_replayable = False

    def launch_key(self, ctx) -> tuple:
        """What this part's launches depend on besides the step's sizes (``ctx.n_tokens``,
        ``n_reqs``, ``n_logit_rows``, ``n_decode``, ``n_tiles``, ``n_tiles_wide``): two steps of a
        model whose parts are all ``launches_replayable``, with equal sizes and equal keys, make
        the same library calls with the same arguments, so the engine may issue a recorded list
        of them again."""
        return ()


def step_decode_plan(part: Part, ctx) -> tuple:
    """How ``part`` cuts the keys of decoded requests in this step: what the engine fixed for a captured step
    (``ctx.extras["decode_plans"]``: a plan per part, by ``id``; or one plan for all, ``"decode_plan"``), else the
    part's own ``decode_plan_for`` the step's sizes."""
    plans = ctx.extras.get("decode_plans")
    if plans is not None and id(part) in plans:
        return plans[id(part)]
    return ctx.extras.get("decode_plan") or part.decode_plan_for(ctx.n_decode, ctx.max_kv_len, ctx.act_dtype)


def build_part(category: str, spec: Any, **extra: Any) -> Part:
    cls = part_class(category, spec.kind)
    return cls(**spec.params, **extra)

"""Differential attention: a head's result is the difference of two softmax maps over the same values.

Built on the windowed attention (``parts/windowed.py``) and its kernels, which keep both maps of a block's rows side
by side so that keys and values are fetched once for the two (csrc/bias_attention.cu, ``maps``).
"""
from __future__ import annotations

import torch

from .base import ParamSpec, register_part
from .windowed import WindowAttention


@register_part("mixer", "differential_attention")
class DifferentialAttention(WindowAttention):
    """``q`` has two vectors a head and ``k`` two a key/value head, laid out head by head as [map 1, map 2]; each is
    rotated by itself (the first ``rot_dims`` entries).  Each map is a softmax of its own over the keys a query sees
    (``window``, ``chunk`` or all earlier ones), both over the head's one value of ``value_dim`` entries:

        lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff            (one number a layer)
        o      = a_1 - lambda a_2,    o <- o / sqrt(mean(o^2) + norm_eps) * (1 - diff)    per head

    and the merged heads through ``W_o``.  lambda depends on weights alone and is worked out once, when they are bound
    (float64, kept in float32).  The cache row of a key/value head is [key 1 | key 2 | value].  ``own_kv=False``: the
    layer has no projections of keys and values and reads another layer's cache, with its own queries, mask, factor
    and scale."""

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, scale: float,
                 norm_eps: float, diff: float, window: int | None = None, chunk: int | None = None, rot_dims: int = 0,
                 rot_base: float = 10000.0, rot_scaling: dict | None = None, own_kv: bool = True) -> None:
        super().__init__(hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale, norm_eps, window=window,
                         rot_dims=rot_dims, rot_base=rot_base, qk_norm=False, unit_values=False, head_temperature=False,
                         rot_scaling=rot_scaling, chunk=chunk, own_kv=own_kv, maps=2)
        self.diff = float(diff)
        self.diff_lambda = None

    def param_specs(self):
        return super().param_specs() + [ParamSpec(r, (self.key_dim,), kind="vector") for r in ("lq1", "lk1", "lq2", "lk2")]

    def bind(self, tensors) -> None:
        super().bind(tensors)
        d = {r: tensors[r].double() for r in ("lq1", "lk1", "lq2", "lk2")}
        lam = torch.exp((d["lq1"] * d["lk1"]).sum()) - torch.exp((d["lq2"] * d["lk2"]).sum()) + self.diff
        self.diff_lambda = lam.to(torch.float32).reshape(1).contiguous()

    def _attention_options(self) -> dict:
        return dict(diff_lambda=self.diff_lambda, diff_eps=self.norm_eps, diff_mul=1.0 - self.diff)

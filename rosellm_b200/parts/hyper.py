"""Hyper-connections: a residual stream kept in several copies, read and written by sublayers with learned weights."""
from __future__ import annotations

import torch

from ..ops import kernels as K
from .base import ParamSpec, Part, register_part
from .standard import RMSNorm


@register_part("connection", "hyper_connection")
class HyperConnection(Part):
    """The weights by which one sublayer reads and writes a stream of ``copies`` copies X_s:

        u = sum_s in_s X_s,    y = sublayer(norm(u)),    X'_t = sum_s mix[s, t] X_s + out_t y

    every new copy from the old ones (``mix`` is indexed [from, to]); float32 in both precisions."""

    graph_safe = True
    launches_replayable = True

    def __init__(self, copies: int) -> None:
        if not 1 <= copies <= K.HYPER_MAX_COPIES:
            raise ValueError(f"hyper-connections: {copies} copies of the stream; 1 to {K.HYPER_MAX_COPIES}")
        self.copies = int(copies)
        self.in_weight = self.out_weight = self.mix = None

    def param_specs(self):
        return [ParamSpec("in_weight", (self.copies,), kind="vector", init="ones"),
                ParamSpec("out_weight", (self.copies,), kind="vector", init="ones"),
                ParamSpec("mix", (self.copies, self.copies), kind="vector", init="eye")]


@register_part("block", "hyper_connections")
class HyperConnectionsBlock(Part):
    """Pre-norm sublayers (a mixer, and a feed-forward where the layer has one) on a stream of several copies, each
    with a ``HyperConnection`` of its own.

    The copies live in a workspace buffer [tokens, copies, width] from the first such layer of a step on: they begin
    as equal copies of the stream's row, which is read as it stands until the first write spreads it.  A sublayer's
    write, the next sublayer's read and the norm ahead of that are one kernel (``K.hyper_step``), also across
    layers, so a layer launches two of them; a mixture of experts leaves its outputs unsummed for that kernel
    (``forward_deferred``).  Behind the last such layer (the layer that runs next is arranged otherwise, or none
    does) the copies' sum becomes the stream's row."""

    graph_safe = True
    launches_replayable = True
    keeps_copies = True

    def __init__(self, copies: int, feed_forward: bool = True) -> None:
        self.copies, self.has_feed_forward = int(copies), bool(feed_forward)
        self.uses = {"norm_mixer": "norm", "mixer": "mixer", "connect_mixer": "connection"}
        if feed_forward:
            self.uses.update(norm_feed_forward="norm", feed_forward="feed_forward", connect_feed_forward="connection")

    def forward(self, ctx, run, layer, x) -> None:
        n, width = x.shape
        ws = ctx.workspace
        kept = ctx.extras.pop("stream_copies", None)  # (the copies, the first norm's output) as the layer before left them
        if kept is None:
            source, h = x, ws.get("hyper_normed", (n, width), ctx.act_dtype)
            K.hyper_step(x, None, copies=self.copies, read=layer.connect_mixer.in_weight, gamma=layer.norm_mixer.weight,
                         eps=layer.norm_mixer.eps, h=h)
        else:
            source, h = kept
        copies = ws.get("hyper_copies", (n, self.copies, width), torch.float32)
        y = ws.get("sublayer_out", (n, width), torch.float32)
        layer.mixer.forward(ctx, run, h, y, add=False)
        last = layer.connect_mixer
        if self.has_feed_forward:
            nxt = layer.connect_feed_forward
            K.hyper_step(source, y, copies=self.copies, write=(last.mix, last.out_weight), x_new=copies, read=nxt.in_weight,
                         gamma=layer.norm_feed_forward.weight, eps=layer.norm_feed_forward.eps, h=h)
            source, last = copies, nxt
            deferred = getattr(layer.feed_forward, "forward_deferred", None)
            if deferred is not None:
                y = deferred(ctx, h)
            else:
                layer.feed_forward.forward(ctx, h, y, add=False)
        follow = ctx.extras.get("next_layer")
        if (follow is not None and isinstance(follow.block, HyperConnectionsBlock) and follow.block.copies == self.copies
                and isinstance(follow.norm_mixer, RMSNorm)):
            K.hyper_step(source, y, copies=self.copies, write=(last.mix, last.out_weight), x_new=copies,
                         read=follow.connect_mixer.in_weight, gamma=follow.norm_mixer.weight, eps=follow.norm_mixer.eps, h=h)
            ctx.extras["stream_copies"] = (copies, h)
        else:
            K.hyper_step(source, y, copies=self.copies, write=(last.mix, last.out_weight), total=x)

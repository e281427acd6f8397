"""Vebotar as a list of parts.

A decoder-only model whose residual stream is kept in several copies (hyper-connections): every sublayer reads a
weighted sum of them, normalised, and writes all of them anew from the old ones and its result.  The mixer is
differential attention over chunks of positions with rotated queries and keys (frequencies stretched along a ramp);
a layer may read the cached keys and values of an earlier one instead of having its own.  The feed-forward is a
mixture of experts with one input projection each (squared relu), chosen by the largest router logits and weighted by
the softmax over the chosen ones, beside a shared expert behind a sigmoid gate; a layer may have none.  The sum of the
copies, an RMS norm and a linear head of its own give the logits.

Tensor names: ``embed``, ``final.norm``, ``head``; layer i: ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.{in,out,mix}``,
``l<i>.hc2.{in,out,mix}``, ``l<i>.mix.{q,k,v,lq1,lk1,lq2,lk2,o}`` (no ``k`` and ``v`` in a layer that reads another's),
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{up,down}``, ``l<i>.mlp.shared.{up,down,sg}``.  Linear weights are stored [out, in].
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.vebotar import VebotarConfig
from ..parts.spec import Concat, LayerSpec, ModelSpec, PartSpec, RunEntry


def _mixer_spec(mx, m: str, width: int, eps: float) -> PartSpec:
    tensors = {"q_weight": m + "q", "out_weight": m + "o", **{r: m + r for r in ("lq1", "lk1", "lq2", "lk2")}}
    if mx.kv_from is None:
        tensors.update(k_weight=m + "k", v_weight=m + "v")
    rot = mx.rot
    return PartSpec(
        "differential_attention",
        dict(hidden_size=width, num_heads=mx.heads, num_kv_heads=mx.kv_heads, key_dim=mx.dim, value_dim=mx.vdim, scale=mx.scale,
             norm_eps=eps, diff=mx.diff, chunk=mx.chunk, rot_dims=0 if rot is None else rot.dims,
             rot_base=10000.0 if rot is None else rot.base, rot_scaling=None if rot is None else rot.scaling_params(),
             own_kv=mx.kv_from is None),
        tensors)


def _feed_forward_spec(mlp, p: str, width: int) -> PartSpec:
    experts = [f"{p}e{j}." for j in range(mlp.experts)]
    tensors = {"router_weight": p + "router", "up_weight": Concat(tuple(e + "up" for e in experts), dim=0),
               "down_weight": Concat(tuple(e + "down" for e in experts), dim=0)}
    if mlp.shared_ff:
        tensors.update(shared_up_weight=p + "shared.up", shared_down_weight=p + "shared.down", shared_gate_weight=p + "shared.sg")
    return PartSpec("moe", dict(hidden_size=width, inner_size=mlp.ff, num_experts=mlp.experts, top=mlp.top, gate="relu_squared",
                                score="chosen_softmax", shared_inner=mlp.shared_ff), tensors)


def build_vebotar_spec(cfg: VebotarConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> tuple[str, PartSpec]:
        return ("norm", PartSpec("rms_norm", dict(hidden_size=width, eps=eps), {"weight": name}))

    def connection(name: str) -> tuple[str, PartSpec]:
        return ("connection", PartSpec("hyper_connection", dict(copies=cfg.streams),
                                       {"in_weight": name + ".in", "out_weight": name + ".out", "mix": name + ".mix"}))

    layers = []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        named = dict(norm_mixer=norm(p + "norm1"), connect_mixer=connection(p + "hc1"),
                     mixer=("mixer", _mixer_spec(lc.mixer, p + "mix.", width, eps)))
        if lc.mlp is not None:
            named.update(norm_feed_forward=norm(p + "norm2"), connect_feed_forward=connection(p + "hc2"),
                         feed_forward=("feed_forward", _feed_forward_spec(lc.mlp, p + "mlp.", width)))
        layers.append(LayerSpec.of(PartSpec("hyper_connections", dict(copies=cfg.streams, feed_forward=lc.mlp is not None)), **named))
    return ModelSpec(
        hidden_size=width,
        vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_table", dict(vocab_size=cfg.vocab, hidden_size=width, scale=cfg.embedding_scale),
                           {"weight": "embed"}),
        position=PartSpec("none"),
        layers=tuple(layers),
        run_order=tuple(RunEntry(i, cache_of=lc.mixer.kv_from) for i, lc in enumerate(cfg.layers)),
        final_norm=PartSpec("rms_norm", dict(hidden_size=width, eps=eps), {"weight": "final.norm"}),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, hidden_size=width), {"weight": "head"}),
        eos_token_id=cfg.eos_token_id,
    )


register_architecture("Vebotar", VebotarConfig, build_vebotar_spec, model_types=("vebotar",), replace=True)

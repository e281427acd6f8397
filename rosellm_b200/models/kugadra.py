"""Kugadra as a list of parts.

A decoder-only model with norms on both sides of every sublayer: ``x += norm1b(mixer(norm1(x)))``, ``x +=
norm2b(ff(norm2(x)))``.  Two mixers, in whatever order the configuration lists them: linear attention whose state decays by
one fixed factor a head, with silu'd queries, keys and values, a norm over the merged heads and an element-wise gate
(``lightning``); and latent attention with a query latent, rotations in halves with ramp-scaled frequencies and a gate per
head (``latent_attention``), which may read the latents that an earlier layer has cached.  Feed-forwards: dense with a
squared relu, or gated experts chosen by the softmax of a router plus a correction, weighted by their shares of the chosen
scores times a factor, beside a shared expert; a layer may have none.  The token rows are scaled on their way into the
stream; final RMS norm; the logits are the embedding table's product, bounded smoothly.

Tensor names: ``embed``, ``final.norm``; layer i: ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``,
``l<i>.mix.*`` (lightning: ``q, k, v, g, norm, o``; latent_attention: ``dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o``, no
``dkv`` and ``dkv.norm`` in a layer that reads another's), ``l<i>.mlp.{up,down}`` or ``l<i>.mlp.{router,correction}`` with
``l<i>.mlp.e<j>.{gate,up,down}`` and ``l<i>.mlp.shared.{gate,up,down}``.  Linear weights are stored [out, in].
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.kugadra import KugadraConfig
from ..parts.spec import Concat, LayerSpec, ModelSpec, PartSpec, RunEntry


def _mixer_spec(kind: str, mx, m: str, width: int, eps: float) -> PartSpec:
    if kind == "lightning":
        return PartSpec("lightning_attention",
                        dict(hidden_size=width, num_heads=mx.heads, key_dim=mx.dim, value_dim=mx.vdim, decay=mx.decay, norm_eps=eps),
                        {"q_weight": m + "q", "k_weight": m + "k", "v_weight": m + "v", "g_weight": m + "g", "out_norm": m + "norm",
                         "out_weight": m + "o"})
    tensors = {"dq_weight": m + "dq", "dq_norm": m + "dq.norm", "q_weight": m + "uq", "uk_weight": m + "uk", "uv_weight": m + "uv",
               "gate_weight": m + "g", "o_weight": m + "o"}
    if mx.kv_from is None:
        tensors.update(dkv_weight=m + "dkv", dkv_norm=m + "dkv.norm")
    return PartSpec(
        "latent_attention",
        dict(hidden_size=width, num_heads=mx.heads, plain_dim=mx.dim, rot_dim=mx.rot_dim, value_dim=mx.vdim, kv_rank=mx.kv_rank,
             scale=mx.scale, rot_dims=mx.rot_dim, rot_base=mx.rot_base, norm_eps=eps, sink=False, q_rank=mx.q_rank, gate="head",
             rot_scaling=mx.scaling_params(), rot_pairs="halves", own_kv=mx.kv_from is None),
        tensors)


def _feed_forward_spec(mlp, p: str, width: int) -> PartSpec:
    if mlp.kind == "dense":
        return PartSpec("dense_mlp", dict(hidden_size=width, inner_size=mlp.ff, activation="relu_squared", bias=False),
                        {"in_weight": p + "up", "out_weight": p + "down"})
    experts = [f"{p}e{j}." for j in range(mlp.experts)]
    tensors = {"router_weight": p + "router", "correction": p + "correction",
               "gate_up_weight": Concat(tuple(e + w for e in experts for w in ("gate", "up")), dim=0),
               "down_weight": Concat(tuple(e + "down" for e in experts), dim=0)}
    if mlp.shared_ff:
        tensors.update(shared_gate_up_weight=Concat((p + "shared.gate", p + "shared.up"), dim=0), shared_down_weight=p + "shared.down")
    return PartSpec("moe", dict(hidden_size=width, inner_size=mlp.ff, num_experts=mlp.experts, top=mlp.top, gate="silu",
                                correction=True, weight_scale=mlp.scale, shared_inner=mlp.shared_ff), tensors)


def build_kugadra_spec(cfg: KugadraConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> tuple[str, PartSpec]:
        return ("norm", PartSpec("rms_norm", dict(hidden_size=width, eps=eps), {"weight": name}))

    layers = []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        named = dict(norm_mixer=norm(p + "norm1"), mixer=("mixer", _mixer_spec(lc.type, lc.mixer, p + "mix.", width, eps)),
                     norm_mixer_out=norm(p + "norm1b"))
        if lc.mlp is not None:
            named.update(norm_feed_forward=norm(p + "norm2"),
                         feed_forward=("feed_forward", _feed_forward_spec(lc.mlp, p + "mlp.", width)),
                         norm_feed_forward_out=norm(p + "norm2b"))
        layers.append(LayerSpec.of(PartSpec("pre_post_norm", dict(feed_forward=lc.mlp is not None)), **named))
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
        head=PartSpec("tied_to_embedding", dict(vocab_size=cfg.vocab, hidden_size=width, soft_cap=cfg.logit_softcap)),
        eos_token_id=cfg.eos_token_id,
        # a layer without a feed-forward runs no norms around it; its file may hold them all the same
        ignored_tensors=tuple(f"l{i}.{n}" for i, lc in enumerate(cfg.layers) if lc.mlp is None for n in ("norm2", "norm2b")),
    )


register_architecture("Kugadra", KugadraConfig, build_kugadra_spec, model_types=("kugadra",), replace=True)

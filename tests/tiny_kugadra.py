"""Small Kugadra configurations for the tests, and helpers to write them as model folders.

They differ from one another in every size and constant and in the order of their layers, and avoid coincidences: key
and value sizes differ, odd, small and large ones; decays from none (1) to all (0); turned parts of none, two and many
entries with and without a ramp, ramps whose ends meet, lie inside and outside the pairs; layers that read the latents of
an earlier one, several of them one layer, with other head counts and sizes than it; experts from one to forty with one,
some or all of them a token, with and without a shared one; layers without a feed-forward; bounds of the logits that bend
them much, little and hardly at all; score scales at which one key takes nearly all the weight.
"""
from __future__ import annotations

import json
import os

import torch

from rosellm_b200.config.kugadra import KugadraConfig
from rosellm_b200.weights import write_model_folder


def linear(heads, dim, vdim, *decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot=None, kv_from=None):
    """``rot``: (base,) or (base, factor, original, fast, slow)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot_dim, "base": rot[0]}
        if len(rot) > 1:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[1:]))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, scale, cap, layers):
    return {"architecture": "Kugadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_softcap": cap, "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


ROT_A, ROT_B, ROT_D = (10000.0, 8.0, 32, 16.0, 2.0), (77.0,), (300000.0, 16.0, 64, 24.0, 1.5)
RAW_A = model(131, 64, 1e-5, 3.0, 2.5, [
    (linear(3, 12, 20, 0.5, 0.93, 0.999), dense(100)),
    (latent(4, 12, 6, 10, 18, 20, 0.9, ROT_A), moe(5, 2, 24, 1.7, 40)),
    (latent(7, 8, 6, 14, 18, 12, 1.3, ROT_A, kv_from=1), None),
    (linear(2, 24, 8, 1.0, 0.0), moe(7, 3, 20, 0.6)),
])
RAW_B = model(300, 96, 1e-6, 1.0, 30.0, [
    (latent(5, 10, 4, 12, 36, 24, 0.8, ROT_B), moe(3, 3, 40, 2.0, 9)),
    (latent(2, 9, 4, 5, 36, 7, 1.1, ROT_B, kv_from=0), dense(72)),
    (linear(7, 9, 5, 0.1, 0.3, 0.6, 0.8, 0.9, 0.97, 0.995), None),
    (latent(3, 40, 4, 8, 36, 44, 0.3, ROT_B, kv_from=0), moe(40, 6, 10, 2.5, 33)),
])
RAW_C = model(77, 48, 1e-4, 0.5, 1.2, [
    (linear(1, 40, 130, 0.98), moe(1, 1, 20, 0.8, 8)),
    (linear(4, 6, 7, 0.9, 0.99, 0.7, 1.0), dense(36)),
    (linear(2, 130, 16, 0.95, 0.4), moe(9, 9, 12, 3.0)),
])
RAW_D = model(2000, 384, 1e-5, 12.5, 6.0, [
    (linear(6, 64, 72, 0.6, 0.8, 0.9, 0.95, 0.98, 0.997), dense(640)),
    (latent(6, 64, 32, 96, 200, 136, 0.2, ROT_D), moe(6, 4, 96, 1.5, 160)),
    (linear(3, 32, 128, 0.75, 0.96, 0.9995), moe(16, 2, 64, 2.2, 88)),
    (latent(12, 24, 32, 24, 200, 72, 0.3, ROT_D, kv_from=1), moe(4, 1, 128, 1.1)),
])
# no turned part at all; one kind of mixer throughout; no feed-forward
RAW_E = model(90, 40, 1e-5, 2.0, 8.0, [
    (latent(5, 8, 0, 8, 16, 16, 0.9), None),
    (latent(3, 20, 0, 6, 16, 9, 0.6, kv_from=0), None),
])
RAW_F = model(64, 56, 1e-5, 7.0, 15.0, [
    (linear(5, 16, 24, 0.85, 0.9, 0.5, 0.99, 0.2), moe(8, 2, 48, 1.3, 72)),
    (latent(8, 12, 10, 16, 40, 28, 2.0, (50.0, 3.0, 24, 6.0, 5.9)), dense(64)),
])
TINY = {
    "A": dict(raw=RAW_A, seed=101, std=0.2, page_size=16),
    "B": dict(raw=RAW_B, seed=102, std=0.15, page_size=8),
    "C": dict(raw=RAW_C, seed=103, std=0.25, page_size=32),
    "D": dict(raw=RAW_D, seed=104, std=0.07, page_size=16),
    "E": dict(raw=RAW_E, seed=105, std=0.3, page_size=16),
    "F": dict(raw=RAW_F, seed=106, std=0.2, page_size=8),
}
# A wide one: the products' tensor-core paths, many chunks, a latent of 256.
ROT_WIDE = (1.0e6, 8.0, 256, 24.0, 2.0)
RAW_WIDE = model(3000, 1024, 1e-5, 4.0, 20.0, [
    (linear(8, 64, 128, *(1.0 - 2.0 ** -(i + 1) for i in range(8))), dense(2048)),
    (latent(16, 64, 32, 64, 256, 384, 0.12, ROT_WIDE), moe(8, 2, 512, 2.0, 1024)),
    (linear(4, 128, 256, 0.7, 0.98, 0.999, 0.9), moe(16, 4, 256, 1.5)),
    (latent(12, 48, 32, 80, 256, 256, 0.15, ROT_WIDE, kv_from=1), moe(8, 2, 512, 1.2, 512)),
])
WIDE = dict(raw=RAW_WIDE, seed=111, std=0.03, page_size=16)


def write_tiny(name: str, root: str, decisive: bool = False) -> str:
    """A model folder of random weights.  Gates are scaled up so that they close and open; the routers' corrections are of
    the scores' own size, so that they change which experts are chosen.
    ``decisive`` (the folders of the 16-bit runs): a layer's experts are near copies of its first (nine parts of it,
    one part their own), so that a choice of experts which is a close call, and which 16-bit rounding turns, changes the
    logits no more than rounding does.  Choices among unlike experts are what the 32-bit runs test."""
    from safetensors.torch import load_file, save_file

    t = WIDE if name == "WIDE" else TINY[name]
    out = os.path.join(root, f"kugadra_{name}" + ("_decisive" if decisive else ""))
    if not os.path.isfile(os.path.join(out, "model.safetensors")):
        write_model_folder(KugadraConfig.from_dict(t["raw"]), t["seed"], out, std=t["std"], norm_affine="random")
        path = os.path.join(out, "model.safetensors")
        tensors = load_file(path)
        g = torch.Generator().manual_seed(t["seed"])
        for key in sorted(tensors):
            old = tensors[key]
            if key.endswith("mlp.correction"):
                tensors[key] = torch.randn(old.shape, generator=g) / old.numel()
            elif key.endswith("mix.g"):
                tensors[key] = (old.float() * 3.0).to(old.dtype)
            elif decisive and ".mlp.e" in key and ".mlp.e0." not in key:
                first = tensors[key[:key.index(".mlp.e")] + ".mlp.e0." + key.rsplit(".", 1)[1]]
                tensors[key] = (0.9 * first.float() + 0.1 * old.float()).to(old.dtype)
        save_file(tensors, path)
    return out


def load_folder(folder: str):
    """The configuration as a dict and the tensors in float64."""
    from safetensors.torch import load_file

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: (v.double() if v.is_floating_point() else v)
                 for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}

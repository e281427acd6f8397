"""Small Vebotar configurations for the tests, and helpers to write them as model folders.

They differ from one another in every size and constant and avoid coincidences: key and value sizes differ, one to
seven query heads a key/value head, turned entries fewer than the key size, all of it or none, odd and large per-head
sizes, chunks of one key, within a page, of a page, across pages, longer than any prompt, or none; one to five copies
of the stream; layers that read another layer's keys and values under the same mask, a smaller one, a larger one or
none, several of them reading one layer; experts from one to forty with one, some or all of them a token; with and
without a shared expert; layers without a feed-forward; ramps whose ends meet, lie inside, and lie outside the pairs.
"""
from __future__ import annotations

import json
import os

import torch

from rosellm_b200.config.vebotar import VebotarConfig
from rosellm_b200.weights import write_model_folder


def attn(heads, kv_heads, dim, vdim, scale, diff, chunk, rot=None, kv_from=None):
    """``rot``: (dims, base) or (dims, base, factor, original, fast, slow)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2:]))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, scale, streams, layers):
    return {"architecture": "Vebotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "streams": streams, "layers": [{"type": "attention", "mixer": m, "mlp": mlp} for m, mlp in layers]}


RAW_A = model(131, 64, 1e-5, 3.0, 3, [
    (attn(6, 2, 16, 24, 0.3, 0.2, 7, (8, 500.0, 4.0, 24, 6.0, 1.0)), moe(5, 2, 24, 40)),
    (attn(6, 2, 16, 24, 0.25, 0.6, 50, (8, 500.0, 4.0, 24, 6.0, 1.0), kv_from=0), moe(7, 3, 20, 12)),
    (attn(4, 4, 24, 8, 0.2, 0.35, 16, (24, 9000.0, 2.0, 64, 8.0, 2.0)), None),
    (attn(4, 4, 24, 8, 0.3, 0.8, 5, (24, 9000.0, 2.0, 64, 8.0, 2.0), kv_from=2), moe(4, 1, 16)),
])
RAW_B = model(300, 96, 1e-6, 1.0, 2, [
    (attn(7, 1, 9, 5, 0.35, 0.1, 33, (6, 77.0)), moe(3, 3, 40, 24)),
    (attn(7, 1, 9, 5, 0.3, 0.5, None, (6, 77.0), kv_from=0), moe(40, 6, 10, 9)),
    (attn(2, 2, 48, 40, 0.14, 0.4, 100, (2, 1.0e6, 16.0, 512, 32.0, 1.0)), moe(6, 2, 28, 36)),
])
RAW_C = model(77, 48, 1e-4, 0.5, 1, [
    (attn(3, 3, 8, 16, 0.4, 0.7, 1, (4, 33.0, 8.0, 20, 4.0, 0.5)), moe(1, 1, 20, 8)),
    (attn(40, 1, 6, 8, 0.4, 0.3, 1000), moe(9, 4, 12, 44)),
])
RAW_D = model(2000, 384, 1e-5, 12.5, 4, [
    (attn(12, 4, 40, 80, 0.15, 0.45, 48, (32, 300000.0, 8.0, 96, 16.0, 1.5)), moe(6, 4, 96, 160)),
    (attn(2, 1, 136, 130, 0.08, 0.25, 128, (136, 5000.0)), moe(16, 2, 64, 88)),
    (attn(12, 4, 40, 80, 0.12, 0.65, 96, (32, 300000.0, 8.0, 96, 16.0, 1.5), kv_from=0), None),
    (attn(12, 4, 40, 80, 0.2, 0.15, 48, (32, 300000.0, 8.0, 96, 16.0, 1.5), kv_from=0), moe(5, 5, 32, 24)),
])
RAW_E = model(90, 40, 1e-5, 2.0, 5, [
    (attn(5, 5, 8, 8, 0.3, 0.5, 32), None),
    (attn(5, 5, 8, 8, 0.3, 0.5, 32, kv_from=0), None),
])
RAW_F = model(64, 56, 1e-5, 7.0, 2, [
    (attn(8, 2, 32, 64, 0.18, 0.55, None, (16, 50.0, 3.0, 24, 6.0, 5.9)), moe(8, 2, 48, 72)),
])
TINY = {
    "A": dict(raw=RAW_A, seed=81, std=0.2, page_size=16),
    "B": dict(raw=RAW_B, seed=82, std=0.15, page_size=8),
    "C": dict(raw=RAW_C, seed=83, std=0.25, page_size=32),
    "D": dict(raw=RAW_D, seed=84, std=0.07, page_size=16),
    "E": dict(raw=RAW_E, seed=85, std=0.3, page_size=16),
    "F": dict(raw=RAW_F, seed=86, std=0.2, page_size=8),
}
# A wide one: the products' tensor-core paths, chunks of many key tiles, two maps of 64 over values of 128.
RAW_WIDE = model(3000, 1024, 1e-5, 4.0, 2, [
    (attn(8, 8, 64, 128, 0.125, 0.3, 300, (32, 1.0e6, 8.0, 256, 24.0, 2.0)), moe(8, 2, 512, 1024)),
    (attn(8, 8, 64, 128, 0.125, 0.6, 300, (32, 1.0e6, 8.0, 256, 24.0, 2.0), kv_from=0), moe(16, 4, 256, 512)),
    (attn(16, 4, 32, 64, 0.18, 0.2, 512, (32, 20000.0)), moe(8, 2, 512)),
])
WIDE = dict(raw=RAW_WIDE, seed=91, std=0.03, page_size=16)


def write_tiny(name: str, root: str, decisive: bool = False) -> str:
    """A model folder of random weights.  The streams' weights are spread around values at which every copy counts (read
    weights of both signs, mixing matrices far from the identity and not symmetric), the factors of the second maps over
    (-1, 2), the shared experts' gates open and close.
    ``decisive`` (the folders of the 16-bit runs): a layer's experts are near copies of its first (nine parts of it,
    one part their own), so that a choice of experts which is a close call, and which 16-bit rounding turns, changes the
    logits no more than rounding does.  Choices among unlike experts are what the 32-bit runs test."""
    from safetensors.torch import load_file, save_file

    t = WIDE if name == "WIDE" else TINY[name]
    out = os.path.join(root, f"vebotar_{name}" + ("_decisive" if decisive else ""))
    if not os.path.isfile(os.path.join(out, "model.safetensors")):
        write_model_folder(VebotarConfig.from_dict(t["raw"]), t["seed"], out, std=t["std"], norm_affine="random")
        path = os.path.join(out, "model.safetensors")
        tensors = load_file(path)
        g = torch.Generator().manual_seed(t["seed"])
        copies = t["raw"]["streams"]
        for key in sorted(tensors):
            old = tensors[key]
            if key.endswith((".hc1.in", ".hc2.in")):
                tensors[key] = 1.0 / copies + 0.4 * torch.randn(old.shape, generator=g)
            elif key.endswith((".hc1.out", ".hc2.out")):
                tensors[key] = 0.8 + 0.4 * torch.randn(old.shape, generator=g)
            elif key.endswith((".hc1.mix", ".hc2.mix")):
                tensors[key] = 0.7 * torch.eye(copies) + 0.3 * torch.randn(old.shape, generator=g) / copies ** 0.5
            elif key.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
                tensors[key] = torch.randn(old.shape, generator=g) * 0.6 / old.numel() ** 0.25
            elif key.endswith("shared.sg"):
                tensors[key] = (old.float() * 4.0).to(old.dtype)
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

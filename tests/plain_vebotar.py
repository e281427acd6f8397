"""A plain, slow implementation of Vebotar: whole sequences, no cache, one function per mechanism.

Written from the design's equations; shares no code with the package.  ``cfg`` is the parsed ``config.json``
(a dict), ``w`` maps tensor names to torch tensors: float64 for the values the tests compare with; given float32
tensors everything is computed in float32, which shows how far rounding alone moves a result.

Notation: ``X`` the streams [S, tokens, width]; ``unit(y) = y / sqrt(mean(y^2) + eps)`` over the last dimension.
A sublayer f with weights a [S], b [S], M [S, S] reads and updates the streams by

    u = sum_s a_s X_s,   y = f(unit(u) * w),   X'_t = sum_s M[s, t] X_s + b_t y      (every t from the old X)

The mixers are differential attentions over chunks: two softmax maps a head over the same values, the second
subtracted with one factor a layer, the difference brought to unit root mean square.  The feed-forwards are
mixtures of experts with a gated shared expert beside them.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

F64 = torch.float64

# Where an engine that keeps activations in 16 bits rounds them (rows that matrix products read, cached keys and
# values, the mixers' results ahead of their output products, inner rows of the feed-forwards): the identity, or a
# function that rounds, to see how far such rounding alone moves the logits of a sequence.
_round = lambda t: t


def to_bfloat16_and_back(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


def unit(y: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


# ---- rotation ---------------------------------------------------------------------------------------------

def ramp_frequencies(dims: int, base: float, scaling: dict | None) -> tuple[list[float], float]:
    """(frequency of every pair, factor of cosines and sines).  Without ``scaling``: base^(-2i/dims) and 1.  With
    it: pairs that turn more than ``fast`` times within ``original`` positions keep their frequency, pairs that turn
    less than ``slow`` times are slowed by ``factor``, between the two the index decides linearly."""
    plain = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(place(float(scaling["fast"]))), 0)
    last = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    width = max(last - first, 0.001)
    out = []
    for i, f in enumerate(plain):
        share = min(max((i - first) / width, 0.0), 1.0)  # 0: kept, 1: slowed
        out.append(share * (f / factor) + (1.0 - share) * f)
    return out, 0.1 * math.log(factor) + 1.0


def turn(y: torch.Tensor, positions: torch.Tensor, freqs: list[float], mult: float) -> torch.Tensor:
    """y [tokens, ..., dim]: neighbouring entries (2i, 2i+1), i < len(freqs), turned by position * freqs[i], with
    cosines and sines times ``mult``; entries beyond them pass unchanged (not even multiplied)."""
    out = y.clone()
    shape = [y.shape[0]] + [1] * (y.dim() - 2)
    for i, f in enumerate(freqs):
        ang = positions.to(y.dtype) * f
        c, s = (torch.cos(ang) * mult).view(shape), (torch.sin(ang) * mult).view(shape)
        a, b = y[..., 2 * i], y[..., 2 * i + 1]
        out[..., 2 * i] = a * c - b * s
        out[..., 2 * i + 1] = b * c + a * s
    return out


# ---- attention --------------------------------------------------------------------------------------------

def seen_keys(T: int, size: int | None) -> torch.Tensor:
    """[T, T] bool: query i (rows) sees key j when j <= i and both lie in the same chunk of ``size`` positions,
    chunks counted from the sequence's first token (``None``: one chunk)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if size is None else ok & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def difference_factor(lq1, lk1, lq2, lk2, diff: float):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def two_maps(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int | None) -> torch.Tensor:
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> [T, H, 2, dv]: every map's own softmax over the keys a query
    sees, both maps of a head over the same values; query head h uses key/value head h // (H / G)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    ok = seen_keys(T, size)
    out = torch.zeros(T, H, 2, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for m in range(2):
            s = (q[:, h, m] @ k[:, g, m].T) * scale
            out[:, h, m] = torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v[:, g]
    return out


def combine_maps(maps: torch.Tensor, lam, diff: float, eps: float) -> torch.Tensor:
    """[..., 2, dv] -> [..., dv]: the difference of the maps, each head at unit root mean square, times 1 - diff."""
    return unit(maps[..., 0, :] - lam * maps[..., 1, :], eps) * (1.0 - diff)


def keys_and_values(h: torch.Tensor, w: dict, p: str, m: dict) -> tuple[torch.Tensor, torch.Tensor]:
    """What a layer that has keys and values of its own caches: turned keys [T, G, 2, d] and values [T, G, dv]."""
    T, G = h.shape[0], m["kv_heads"]
    k = (h @ w[p + "k"].T).view(T, G, 2, m["dim"])
    v = (h @ w[p + "v"].T).view(T, G, m["vdim"])
    if m.get("rot"):
        k = turn(k, torch.arange(T), *ramp_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling")))
    return _round(k), _round(v)


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, caches: dict, i: int) -> torch.Tensor:
    """``caches``: layer -> (keys, values) of the layers that have run; a layer with ``kv_from`` reads another's."""
    T, h = h.shape[0], _round(h)
    H, d = m["heads"], m["dim"]
    q = (h @ w[p + "q"].T).view(T, H, 2, d)
    if m.get("rot"):
        q = turn(q, torch.arange(T), *ramp_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling")))
    src = m.get("kv_from")
    if src is None:
        caches[i] = keys_and_values(h, w, p, m)
    k, v = caches[i if src is None else src]
    lam = difference_factor(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    size = m["mask"]["size"] if m.get("mask") else None
    o = combine_maps(two_maps(q, k, v, m["scale"], size), lam, m["diff"], eps)
    return _round(o.reshape(T, -1)) @ w[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------

def squared_relu_mlp(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor, gate=1.0) -> torch.Tensor:
    """W_down relu(W_up h)^2, times ``gate`` (a number, or one a token [T, 1])."""
    a = torch.clamp(h @ up.T, min=0.0)
    return _round(a * a * gate) @ down.T


def route(z: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """z [T, E] -> (the ``top`` experts with the largest logits, the softmax over their logits alone)."""
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, -1)


def experts(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    h = _round(h)
    idx, weight = route(h @ w[p + "router"].T, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, c = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += weight[t, c, None] * squared_relu_mlp(h[t], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    if mlp.get("shared"):
        gate = torch.sigmoid(h @ w[p + "shared.sg"].T)
        out = out + squared_relu_mlp(h, w[p + "shared.up"], w[p + "shared.down"], gate)
    return out


# ---- streams and the model --------------------------------------------------------------------------------

def read_streams(X: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    return (a[:, None, None] * X).sum(0)


def write_streams(X: torch.Tensor, M: torch.Tensor, b: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """M is indexed [from, to]."""
    out = torch.zeros_like(X)
    for t in range(X.shape[0]):
        for s in range(X.shape[0]):
            out[t] += M[s, t] * X[s]
        out[t] += b[t] * y
    return out


def sublayer(X: torch.Tensor, w: dict, i: int, q: int, eps: float, f) -> torch.Tensor:
    p = f"l{i}.hc{q}."
    u = read_streams(X, w[p + "in"])
    y = f(unit(u, eps) * w[f"l{i}.norm{q}"])
    return write_streams(X, w[p + "mix"], w[p + "out"], y)


def layer(X: torch.Tensor, w: dict, i: int, lc: dict, eps: float, caches: dict) -> torch.Tensor:
    X = sublayer(X, w, i, 1, eps, lambda h: attention(h, w, f"l{i}.mix.", lc["mixer"], eps, caches, i))
    if lc.get("mlp") is not None:
        X = sublayer(X, w, i, 2, eps, lambda h: experts(h, w, f"l{i}.mlp.", lc["mlp"]))
    return X


def forward(cfg: dict, w: dict, tokens, rounding=None, streams: list | None = None) -> torch.Tensor:
    """Logits [tokens, vocab] of one sequence.  ``streams`` (a list) receives the sum of the streams after every
    layer."""
    global _round
    keep, _round = _round, (rounding or (lambda t: t))
    try:
        eps = cfg["norm"]["eps"]
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
        X = x[None].repeat(cfg["streams"], 1, 1)
        caches: dict = {}
        for i, lc in enumerate(cfg["layers"]):
            X = layer(X, w, i, lc, eps, caches)
            if streams is not None:
                streams.append(X.sum(0))
        return _round(unit(X.sum(0), eps) * w["final.norm"]) @ w["head"].T
    finally:
        _round = keep


# ---- model folders ----------------------------------------------------------------------------------------

_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, m in meta.items():
        if name != "__metadata__":
            a, b = m["data_offsets"]
            out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=_DTYPES[m["dtype"]]).reshape(m["shape"]).clone()
    return out


def load_folder(folder: str, dtype: torch.dtype = F64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in
         read_safetensors(os.path.join(folder, "model.safetensors")).items()}
    return cfg, w

"""A plain, slow implementation of Kugadra: whole sequences, no cache, one function per mechanism.

Written from the design's equations; shares no code with the package.  ``cfg`` is the parsed ``config.json``
(a dict), ``w`` maps tensor names to torch tensors: float64 for the values the tests compare with; given float32
tensors everything is computed in float32, which shows how far rounding alone moves a result.

Notation: ``x`` the stream [tokens, width]; ``norm(y, g) = g * y / sqrt(mean(y^2) + eps)`` over the last dimension.
A layer: ``x <- x + norm1b(mixer(norm1(x)))``, then (where it has one) ``x <- x + norm2b(ff(norm2(x)))``.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

F64 = torch.float64

# Where an engine that keeps activations in 16 bits rounds them (rows that matrix products read, cached latents, the
# linear attention's queries, keys and values, the mixers' results ahead of their output products, inner rows of the feed-forwards): the identity, or a function that
# rounds, to see how far such rounding alone moves the logits of a sequence.
_round = lambda t: t


def to_bfloat16_and_back(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


def norm(y: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * gain


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ---- the linear attention with a fixed decay a head ---------------------------------------------------------

def decayed_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay, state: torch.Tensor | None = None):
    """q, k [T, H, dk], v [T, H, dv]; per head S_t = decay_h S_(t-1) + k_t v_t^T (S_0 = ``state`` or zero) and
    o_t = S_t^T q_t.  Returns o [T, H, dv] and the last state [H, dk, dv]."""
    T, H = q.shape[0], q.shape[1]
    d = torch.as_tensor(decay, dtype=q.dtype).view(H, 1, 1)
    S = torch.zeros(H, q.shape[-1], v.shape[-1], dtype=q.dtype) if state is None else state.to(q.dtype).clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def lightning(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """silu on all three projections; the merged heads' norm is over all of their columns together; gate; output."""
    T, h = h.shape[0], _round(h)
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q, k = (_round(silu(h @ w[p + n].T)).view(T, H, dk) for n in ("q", "k"))
    v = _round(silu(h @ w[p + "v"].T)).view(T, H, dv)
    o, _ = decayed_states(q, k, v, m["decay"])
    o = norm(o.reshape(T, H * dv), w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return _round(o) @ w[p + "o"].T


# ---- rotation -------------------------------------------------------------------------------------------------

def rotation_constants(rot: dict) -> tuple[list[float], float]:
    """(frequency of every pair, factor of cosines and sines) from a mixer's ``rot`` entry; with ``scaling`` a linear
    ramp over the pairs' indices between plain frequencies and frequencies slowed by ``factor``."""
    dims, base = rot["dims"], float(rot["base"])
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freqs, 1.0

    def index_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(y: torch.Tensor, positions: torch.Tensor, freqs: list[float], mult: float = 1.0) -> torch.Tensor:
    """y [tokens, ..., dim]: entry i of the first 2 n entries is turned with entry i + n (n = len(freqs)) by position *
    freqs[i]; cosines and sines times ``mult``; further entries pass."""
    out, n = y.clone(), len(freqs)
    shape = [y.shape[0]] + [1] * (y.dim() - 2)
    for i, f in enumerate(freqs):
        ang = positions.to(y.dtype) * f
        c, s = (torch.cos(ang) * mult).view(shape), (torch.sin(ang) * mult).view(shape)
        a, b = y[..., i], y[..., i + n]
        out[..., i] = a * c - b * s
        out[..., i + n] = b * c + a * s
    return out


# ---- latent attention --------------------------------------------------------------------------------------------

def latent_rows(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """What a layer caches of every token: the normed latent [T, kv_rank] and the turned key part [T, rot_dim]."""
    dkv, rank = _round(h) @ w[p + "dkv"].T, m["kv_rank"]
    c = norm(dkv[:, :rank], w[p + "dkv.norm"], eps)
    k_rot = dkv[:, rank:]
    if m.get("rot"):
        freqs, mult = rotation_constants(dict(m["rot"], dims=m["rot_dim"]))
        k_rot = rotate_halves(k_rot, torch.arange(h.shape[0]), freqs, mult)
    return _round(c), _round(k_rot)


def latent_queries(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """Every head's query: the part that meets projected latents [T, H, dim] and the turned part [T, H, rot_dim]."""
    T, h, dn, dr = h.shape[0], _round(h), m["dim"], m["rot_dim"]
    cq = _round(norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps))
    q = (cq @ w[p + "uq"].T).view(T, m["heads"], dn + dr)
    q_rot = q[..., dn:]
    if m.get("rot"):
        freqs, mult = rotation_constants(dict(m["rot"], dims=dr))
        q_rot = rotate_halves(q_rot, torch.arange(T), freqs, mult)
    return q[..., :dn], q_rot


def latent_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, rows) -> torch.Tensor:
    """``rows``: the (latent, turned key part) of this layer or of the layer it names.  Keys and values are projected
    from the latent; plain softmax over all keys up to the query; head h's result times sigmoid((W_g h)_h)."""
    T, H, dn, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c, k_rot = rows
    q_plain, q_rot = latent_queries(h, w, p, m, eps)
    k_plain = (c @ w[p + "uk"].T).view(T, H, dn)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        s = (q_plain[:, hd] @ k_plain[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]
        out[:, hd] = torch.softmax(s.masked_fill(later, -math.inf), -1) @ v[:, hd]
    out = out * torch.sigmoid(_round(h) @ w[p + "g"].T)[:, :, None]
    return _round(out.reshape(T, H * dv)) @ w[p + "o"].T


# ---- feed-forwards ---------------------------------------------------------------------------------------------

def dense(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return _round(torch.clamp(_round(h) @ w[p + "up"].T, min=0.0) ** 2) @ w[p + "down"].T


def gated(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    h = _round(h)
    return _round(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(z: torch.Tensor, correction: torch.Tensor, top: int, scale: float) -> tuple[list[int], torch.Tensor]:
    """One token's experts and their weights from its router logits: the ``top`` largest of softmax(z) + correction;
    the softmax's entries of the chosen, divided by their sum (+ 1e-20), times ``scale``."""
    s = torch.softmax(z, -1)
    ids = torch.argsort(s + correction, descending=True, stable=True)[:top]
    return ids.tolist(), s[ids] / (s[ids].sum() + 1e-20) * scale


def experts(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    z = _round(h) @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, weights = choose(z[t], w[p + "correction"], r["top"], r["scale"])
        for e, a in zip(ids, weights):
            out[t] += a * gated(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + gated(h, w, p + "shared.")
    return out


def feed_forward(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    return dense(h, w, p) if mlp["kind"] == "dense" else experts(h, w, p, mlp)


# ---- the model --------------------------------------------------------------------------------------------------

def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def forward(cfg: dict, w: dict, tokens, rounding=None, streams: list | None = None) -> torch.Tensor:
    """Logits [tokens, vocab] of one sequence.  ``streams`` (a list) receives the stream after every layer."""
    global _round
    keep, _round = _round, (rounding or (lambda t: t))
    try:
        eps = cfg["norm"]["eps"]
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
        cached = {}
        for i, lc in enumerate(cfg["layers"]):
            p, m = f"l{i}.", lc["mixer"]
            h = norm(x, w[p + "norm1"], eps)
            if lc["type"] == "lightning":
                y = lightning(h, w, p + "mix.", m, eps)
            else:
                j = m.get("kv_from")
                if j is None:
                    j, cached[i] = i, latent_rows(h, w, p + "mix.", m, eps)
                y = latent_attention(h, w, p + "mix.", m, eps, cached[j])
            x = x + norm(y, w[p + "norm1b"], eps)
            if lc.get("mlp") is not None:
                h = norm(x, w[p + "norm2"], eps)
                x = x + norm(feed_forward(h, w, p + "mlp.", lc["mlp"]), w[p + "norm2b"], eps)
            if streams is not None:
                streams.append(x.clone())
        z = _round(norm(x, w["final.norm"], eps)) @ w["embed"].T
        return soft_cap(z, cfg["logit_softcap"])
    finally:
        _round = keep


# ---- model folders ------------------------------------------------------------------------------------------------

_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}


def read_safetensors(path: str) -> dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        a, b = m["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=_DTYPES[m["dtype"]]).reshape(m["shape"]).clone()
    return out


def load_folder(folder: str, dtype: torch.dtype = F64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in
         read_safetensors(os.path.join(folder, "model.safetensors")).items()}
    return cfg, w

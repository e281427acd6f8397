"""Kugadra on the GPU: every mechanism's kernels against the plain implementation's function for it, then whole
models through the engine's step function, cache, scheduler and entry point."""
import os
import types

import numpy as np
import pytest
import torch

import plain_kugadra as P
import replay_util as R
from tiny_kugadra import TINY, WIDE, load_folder, write_tiny

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def K():
    from rosellm_b200.ops import kernels

    return kernels


def rel(a: torch.Tensor, b: torch.Tensor) -> float:
    return float((a.double().cpu() - b.double().cpu()).abs().max() / (b.double().abs().max() + 1e-30))


def dev(a):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV)


def to16(t):
    return t.to(torch.bfloat16).to(t.dtype)


# ---- the linear attention with a fixed decay a head ------------------------------------------------------------

def _lightning_step(proj, offsets, powers, state, hb, H, dk, dv, silu, cores):
    n, tiles = len(hb.positions), len(hb.tiles_wide)
    chunks = torch.full((max(tiles, 1) * H * dk * dv,), float("nan"), device=DEV)
    out = torch.full((n, H * dv), float("nan"), device=DEV)
    K().lightning(proj, offsets, powers, state, dev(hb.q_start), dev(hb.slots), chunks if tiles else None, out, n_heads=H, dk=dk, dv=dv,
                  tiles=dev(hb.tiles_wide.reshape(-1)), n_tiles=tiles, decode_reqs=dev(hb.decode_reqs), n_decode=len(hb.decode_reqs),
                  silu=silu, tensor_cores=cores)
    return out


def _lightning_case(H, dk, dv, lens, cuts, seed, *, decays=None, silu=True, cores=False, mark=None):
    """Requests of ``lens`` tokens brought in steps of ``cuts`` tokens in turn (all requests of a step together, a padding
    row of slot -1 beside them), each beginning from a state of its own; ``mark``: (request, token, factor), a token whose
    key and value are scaled.  Largest relative difference of outputs and last states from the plain recurrence."""
    from rosellm_b200.engine.context import build_host_batch

    g = torch.Generator().manual_seed(seed)
    n_req = len(lens)
    d = torch.linspace(0.3, 0.999, H).tolist() if decays is None else decays
    powers = torch.tensor([[x ** n for n in range(65)] for x in d], dtype=torch.float64).float()
    # the projections lie somewhere in a wider matrix, at columns that are multiples of 8
    pad8 = lambda x: -(-x // 8) * 8
    offsets = {"k": 8, "q": 8 + pad8(H * dk) + 16, "v": 8 + 2 * pad8(H * dk) + 16}
    width = offsets["v"] + pad8(H * dv) + 8
    rows = [torch.randn(n, width, generator=g) for n in lens]
    if mark is not None:
        r, t, f = mark
        rows[r][t, offsets["k"]:offsets["k"] + H * dk] = rows[r][t, offsets["k"]:offsets["k"] + H * dk].abs() * f
        rows[r][t, offsets["v"]:offsets["v"] + H * dv] = rows[r][t, offsets["v"]:offsets["v"] + H * dv].abs() * f
    if cores and not silu:  # nothing is lost when they become operands
        rows = [to16(x) for x in rows]
    first = torch.randn(n_req + 2, H, dk, dv, generator=g) * 0.3
    state = first.to(DEV).clone()
    outs = [torch.zeros(n, H * dv) for n in lens]
    at, k = [0] * n_req, 0
    while any(a < n for a, n in zip(at, lens)):
        ents, used = [], []
        for r in range(n_req):
            n = min(cuts[(k + r) % len(cuts)], lens[r] - at[r])
            if n > 0:
                ents.append((r + 1, at[r], [0] * n, []))
                used.append((r, n))
        k += 1
        ents.append((-1, 0, [0], []))
        hb = build_host_batch(ents)
        proj = torch.cat([rows[r][at[r]:at[r] + n] for r, n in used] + [torch.randn(1, width, generator=g)]).to(DEV)
        out = _lightning_step(proj, offsets, powers.to(DEV), state, hb, H, dk, dv, silu, cores).cpu()
        t0 = 0
        for r, n in used:
            outs[r][at[r]:at[r] + n] = out[t0:t0 + n]
            at[r] += n
            t0 += n
        assert torch.isfinite(out).all() and not out[-1].any()
    act = P.silu if silu else (lambda z: z)
    worst = 0.0
    for r in range(n_req):
        q, k_, v = (act(rows[r][:, offsets[n]:offsets[n] + H * w].double()).view(-1, H, w) for n, w in (("q", dk), ("k", dk), ("v", dv)))
        if cores:  # the tensor cores' operands (a single token's are not rounded)
            q, k_, v = to16(q), to16(k_), to16(v)
        want, last = P.decayed_states(q, k_, v, d, first[r + 1].double())
        worst = max(worst, rel(outs[r].view(-1, H, dv), want), rel(state[r + 1], last))
    assert torch.equal(state[0].cpu(), first[0]) and torch.equal(state[n_req + 1].cpu(), first[n_req + 1])  # no one else's state
    return worst


SHAPES = [(3, 12, 20), (1, 40, 130), (7, 9, 5), (2, 130, 16), (6, 64, 72), (4, 16, 256), (1, 256, 64), (2, 1, 1), (5, 33, 3)]


@pytest.mark.parametrize("H,dk,dv", SHAPES)
@pytest.mark.parametrize("silu", [True, False])
def test_decayed_states_in_float32(H, dk, dv, silu):
    """Whole portions around the chunks' edges, portions of every small size, single tokens (states read and written by
    the kernel for them), and mixtures of the two in one step."""
    for lens, cuts in (([1, 2, 63, 64, 65, 128, 130, 200], (1000,)), ([40, 3, 70], (1,)), ([100, 64, 9], (2,)),
                       ([150, 31, 66], (7, 1, 64, 2, 1, 33))):
        assert _lightning_case(H, dk, dv, lens, cuts, seed=H * dk, silu=silu) < 2e-5, (lens, cuts)


@pytest.mark.parametrize("H,dk,dv", SHAPES + [(8, 64, 128), (2, 128, 200)])
def test_decayed_states_on_the_tensor_cores(H, dk, dv):
    """Queries, keys and values are bfloat16 operands; scores, decayed keys and states lose nothing to it beyond what two
    bfloat16 numbers in place of a float32 one lose: on operands that rounding leaves alone the recurrence is met closely,
    with silu ahead of the rounding as closely as 16-bit operands allow."""
    for lens, cuts in (([1, 2, 63, 64, 65, 128, 130, 200], (1000,)), ([100, 64, 9], (2,)), ([150, 31, 66], (7, 1, 64, 2, 1, 33))):
        assert _lightning_case(H, dk, dv, lens, cuts, seed=H * dv, silu=False, cores=True) < 1e-4, (lens, cuts)
        assert _lightning_case(H, dk, dv, lens, cuts, seed=H * dv, cores=True) < 1e-2, (lens, cuts)


@pytest.mark.parametrize("cores", [False, True])
def test_decays_from_all_to_none(cores):
    """Heads that forget at once (0), at once but for a trace, hardly at all and never (1), over 700 tokens; whole against
    portions."""
    d = [0.0, 1e-3, 0.5, 0.97, 0.9999, 1.0]
    for cuts in ((1000,), (5, 2, 90), (64, 128, 65)):
        assert _lightning_case(6, 16, 24, [700, 2, 129], cuts, seed=5, decays=d, silu=not cores, cores=cores) < (1e-4 if cores else 3e-5), cuts


@pytest.mark.parametrize("cores", [False, True])
@pytest.mark.parametrize("token", [0, 1, 62, 63, 64, 65, 127, 128, 640])
def test_a_token_that_stands_out_at_a_chunks_edge_and_far_back(cores, token):
    """One token's key and value are thirty times as large: 900 tokens on, its part of the state is still most of the
    output; the plain result without it is another one."""
    d = [0.9995, 0.999]
    for cuts in ((1000,), (64,), (63, 2, 200)):
        assert _lightning_case(2, 16, 24, [900], cuts, seed=token, decays=d, silu=not cores, cores=cores,
                               mark=(0, token, 30.0)) < (1e-4 if cores else 3e-5), cuts
    g = torch.Generator().manual_seed(token)
    q, k, v = (torch.randn(900, 2, w, generator=g).double() for w in (16, 16, 24))
    k[token], v[token] = k[token].abs() * 30, v[token].abs() * 30
    with_it = P.decayed_states(q, k, v, d)[0][-1]
    v[token] = 0
    assert float((P.decayed_states(q, k, v, d)[0][-1] - with_it).norm() / with_it.norm()) > 0.5


def test_refused_linear_attention():
    z = torch.zeros(4, 64, device=DEV)
    pw, st, out = torch.zeros(1, 65, device=DEV), torch.zeros(2, 1, 8, 8, device=DEV), torch.zeros(4, 8, device=DEV)
    i32 = torch.zeros(4, dtype=torch.int32, device=DEV)
    ok = dict(n_heads=1, dk=8, dv=8, tiles=i32, n_tiles=0, decode_reqs=i32, n_decode=0)
    K().lightning(z, {"q": 0, "k": 8, "v": 16}, pw, st, i32, i32, None, out, **ok)
    for offsets, powers, state, kw in (({"q": 0, "k": 8, "v": 60}, pw, st, {}), ({"q": 0, "k": 8, "v": 16}, pw[:, :64], st, {}),
                                       ({"q": 0, "k": 8, "v": 16}, pw, st[:, :, :4], {})):
        with pytest.raises(K().KernelError):
            K().lightning(z, offsets, powers, state, i32, i32, None, out, **dict(ok, **kw))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [4, 5, 60, 512, 1000, 1023, 2048, 5000])
def test_norm_and_gate_of_the_merged_heads(dtype, width):
    g = torch.Generator().manual_seed(width)
    n, eps = 9, 1e-3
    x, z = torch.randn(n, width + 4, generator=g) * 3, torch.randn(n, width + 12, generator=g) * 4
    gamma = 1 + 0.3 * torch.randn(width, generator=g)
    out = torch.full((n, -(-width // 8) * 8), 7.0, dtype=DTYPES[dtype], device=DEV)
    K().rmsnorm_gate(x.to(DEV)[:, :width], z.to(DEV)[:, 8:8 + width], gamma.to(DEV), eps, out[:, :width])
    want = P.norm(x[:, :width].double(), gamma.double(), eps) * torch.sigmoid(z[:, 8:8 + width].double())
    assert rel(out[:, :width].float(), want) < (2e-6 if dtype == "float32" else 6e-3)
    assert out[:, width:].eq(7.0).all()


# ---- latent attention: gates per head, halves, rows of another layer ---------------------------------------------

class _Cache:
    """One layer's pool of latent rows for a few requests, all pages in place in a random order."""

    def __init__(self, n_req, tokens, page, row, dtype, seed):
        g = torch.Generator().manual_seed(seed)
        per = -(-tokens // page)
        self.pool = torch.full((n_req * per + 2, 1, 1, page, row), 9.0, dtype=dtype, device=DEV)
        self.table = torch.full((n_req + 1, per), -1, dtype=torch.int32)
        self.table[1:] = torch.randperm(n_req * per, generator=g).view(n_req, per)
        self.table = self.table.to(DEV)
        self.device, self.max_seq_len = torch.device(DEV), tokens

    def kv_pool(self, key):
        return self.pool

    def block_table(self, key):
        return self.table


def _latent_part(cfg, width, eps, tensors, dt):
    from rosellm_b200.models.kugadra import _mixer_spec
    from rosellm_b200.config.kugadra import LatentConfig
    from rosellm_b200.parts.base import build_part

    ps = _mixer_spec("latent_attention", LatentConfig.from_dict(cfg, "m"), "", width, eps)
    part = build_part("mixer", ps)
    part.bind({p.role: tensors[ps.tensors[p.role]].to(torch.float32 if p.kind == "vector" else dt).to(DEV).contiguous()
               for p in part.param_specs()})
    return part


def _latent_tensors(cfg, width, seed, std=0.3):
    g = torch.Generator().manual_seed(seed)
    H, dn, dr, dv, r, qr = (cfg[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    shapes = {"dq": (qr, width), "dq.norm": (qr,), "uq": (H * (dn + dr), qr), "dkv": (r + dr, width), "dkv.norm": (r,),
              "uk": (H * dn, r), "uv": (H * dv, r), "g": (H, width), "o": (width, H * dv)}
    out = {}
    for name, s in shapes.items():
        t = torch.randn(s, generator=g) * std
        out[name] = to16(1 + 0.5 * t if name.endswith("norm") else (t * 4 if name == "g" else t))
    return out


class _Run:
    cache_key = state_key = 0

    def __init__(self, writes):
        self.writes_cache = writes


LATENTS = [dict(heads=4, dim=12, rot_dim=6, vdim=10, kv_rank=18, q_rank=20, scale=0.5),
           dict(heads=7, dim=9, rot_dim=10, vdim=5, kv_rank=36, q_rank=7, scale=0.8),
           dict(heads=12, dim=64, rot_dim=32, vdim=96, kv_rank=200, q_rank=136, scale=0.1),
           dict(heads=2, dim=20, rot_dim=0, vdim=24, kv_rank=16, q_rank=9, scale=0.6)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", range(len(LATENTS)))
def test_latent_layers_with_and_without_rows_of_their_own(dtype, which):
    """The part itself: requests in portions (cut inside pages) and single tokens, in one batch; then a second layer of
    other head counts and sizes reads the first's rows, whose pages it must leave alone."""
    from rosellm_b200.engine.context import Workspace, standalone_context

    dt, width, eps = DTYPES[dtype], 48, 1e-5
    own = dict(LATENTS[which])
    if own["rot_dim"]:
        own["rot"] = {"dims": own["rot_dim"], "base": 300.0, "scaling": {"factor": 4.0, "original": 40, "fast": 8.0, "slow": 1.0}}
    reader = dict(own, heads=own["heads"] + 1, dim=own["dim"] + 5, vdim=own["vdim"] + 8, q_rank=own["q_rank"] + 3, kv_from=0)
    tens = [_latent_tensors(c, width, 10 * which + i) for i, c in enumerate((own, reader))]
    parts = [_latent_part(c, width, eps, t, dt) for c, t in zip((own, reader), tens)]
    g = torch.Generator().manual_seed(which)
    lens = [70, 33, 5]
    hs = [[torch.randn(n, width, generator=g).to(dt) for n in lens] for _ in range(2)]  # each layer has an input of its own
    cache = _Cache(len(lens), 80, 16, parts[0].row_width, dt, which)
    assert parts[0].row_width == parts[1].row_width and parts[1].dkv_weight is None
    got = [[torch.zeros(n, width) for n in lens] for _ in range(2)]
    at, step = [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        used = [(r, min((17, 1, 2, 30, 1)[(step + r) % 5], lens[r] - at[r])) for r in range(len(lens)) if at[r] < lens[r]]
        step += 1
        ctx = standalone_context(cache, [(r + 1, at[r], [0] * n, []) for r, n in used], dt, Workspace(torch.device(DEV)))
        for layer, part in enumerate(parts):
            before = cache.pool.clone()
            h = torch.cat([hs[layer][r][at[r]:at[r] + n] for r, n in used]).to(DEV)
            x = torch.full((h.shape[0], width), 3.0, device=DEV)
            part.forward(ctx, _Run(layer == 0), h, x, add=layer == 0)
            assert layer == 0 or torch.equal(before, cache.pool)
            t0 = 0
            for r, n in used:
                got[layer][r][at[r]:at[r] + n] = x[t0:t0 + n].cpu() - (3.0 if layer == 0 else 0.0)
                t0 += n
        for r, n in used:
            at[r] += n
    K().check_status(torch.device(DEV))
    for r, n in enumerate(lens):
        w = [{k: v.double() for k, v in t.items()} for t in tens]
        rows = P.latent_rows(hs[0][r].double(), w[0], "", own, eps)
        for layer, (c, ww) in enumerate(((own, w[0]), (reader, w[1]))):
            want = P.latent_attention(hs[layer][r].double(), ww, "", c, eps, rows)
            assert rel(got[layer][r], want) < (5e-5 if dtype == "float32" else 3e-2), (layer, r)
    with pytest.raises(ValueError):
        parts[1].forward(ctx, _Run(True), h, x)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", [0, 15, 16, 512, 897])
def test_a_key_that_stands_out_far_back(dtype, key):
    """Queries and keys share their projections but for a reordering of the input, so a token points hard at the one whose
    input it holds reordered: as the sequence's first, at pages' borders and hundreds back, from a portion's last query and from a decoded token, through
    the layer's own rows and through those of another layer."""
    from rosellm_b200.engine.context import Workspace, standalone_context

    dt, width, eps, T = DTYPES[dtype], 64, 1e-5, 900
    cfg = dict(heads=3, dim=16, rot_dim=4, vdim=12, kv_rank=24, q_rank=24, scale=1.5, rot={"dims": 4, "base": 50.0})
    t = _latent_tensors(cfg, width, key)
    order = torch.randperm(width, generator=torch.Generator().manual_seed(key + 1))
    t["dq"], t["dq.norm"] = t["dkv"][:24][:, order].clone(), t["dkv.norm"].clone()
    t["uq"].view(3, 20, 24)[:, :16] = t["uk"].view(3, 16, 24)
    t["uq"].view(3, 20, 24)[:, 16:] = 0.01
    t["g"] = t["g"] * 0.0
    g = torch.Generator().manual_seed(key)
    h = torch.randn(T, width, generator=g).to(dt)
    h[T - 1] = h[key][order]
    own, reader = _latent_part(cfg, width, eps, t, dt), _latent_part(dict(cfg, kv_from=0), width, eps, t, dt)
    w = {k: v.double() for k, v in t.items()}
    rows = P.latent_rows(h.double(), w, "", cfg, eps)
    want = P.latent_attention(h.double(), w, "", cfg, eps, rows)[-1]
    c = rows[0].clone()
    c[key] = c[(key + 7) % T]
    assert rel(P.latent_attention(h.double(), w, "", cfg, eps, (c, rows[1]))[-1], want) > 0.2  # its value is most of the result
    for new in (1, 4, 70):
        cache = _Cache(1, T, 16, own.row_width, dt, new)
        ws = Workspace(torch.device(DEV))
        x = torch.zeros(T - new, width, device=DEV)
        own.forward(standalone_context(cache, [(1, 0, [0] * (T - new), [])], dt, ws), _Run(True), h[:T - new].to(DEV), x)
        ctx = standalone_context(cache, [(1, T - new, [0] * new, [])], dt, ws)
        for part in (own, reader):
            x = torch.zeros(new, width, device=DEV)
            part.forward(ctx, _Run(part is own), h[T - new:].to(DEV), x, add=False)
            assert rel(x[-1], want) < (5e-5 if dtype == "float32" else 3e-2), (new, part is own)
    K().check_status(torch.device(DEV))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gate_per_head_on_the_value_product(dtype):
    """One logit a head, read out of a wider matrix; heads of odd sizes too."""
    g = torch.Generator().manual_seed(4)
    for n, H, k, m in ((5, 3, 18, 10), (70, 16, 64, 64), (33, 7, 9, 5)):
        a, w = torch.randn(n, H, k, generator=g).to(DTYPES[dtype]), torch.randn(H, m, k, generator=g).to(DTYPES[dtype])
        z = torch.randn(n, H + 9, generator=g) * 3
        out = torch.zeros(n, H, m, dtype=DTYPES[dtype], device=DEV)
        zd = z.to(DEV)
        K().head_linear(a.to(DEV), w.to(DEV), out, n_tokens=n, n_heads=H, k=k, n=m, in_strides=(H * k, k), w_strides=(m * k, 1, k),
                        out_strides=(H * m, m), gate=zd[:, 5:5 + H], gate_strides=(zd.stride(0), 1, 0))
        want = torch.einsum("thk,hmk->thm", a.double(), w.double()) * torch.sigmoid(z[:, 5:5 + H].double())[:, :, None]
        assert rel(out.float(), want) < (1e-5 if dtype == "float32" else 8e-3)


# ---- experts ---------------------------------------------------------------------------------------------------

def _expert_case(dtype, E, top, n, ff, shared, scale, hid=48, seed=0):
    from rosellm_b200.engine.context import Workspace
    from rosellm_b200.parts.gated import MixtureOfExperts

    g = torch.Generator().manual_seed(seed + E * 7 + top)
    dt = DTYPES[dtype]
    part = MixtureOfExperts(hidden_size=hid, inner_size=ff, num_experts=E, top=top, gate="silu", correction=True, weight_scale=scale,
                            shared_inner=shared)
    t = {"router_weight": torch.randn(E, hid, generator=g) * 0.4, "correction": torch.randn(E, generator=g) / E,
         "gate_up_weight": torch.randn(E * 2 * ff, hid, generator=g) * 0.3, "down_weight": torch.randn(E * hid, ff, generator=g) * 0.3}
    if shared:
        t.update(shared_gate_up_weight=torch.randn(2 * shared, hid, generator=g) * 0.3, shared_down_weight=torch.randn(hid, shared, generator=g) * 0.3)
    t = {k: v if k == "correction" else to16(v) for k, v in t.items()}
    w = {"m.router": t["router_weight"].double(), "m.correction": t["correction"].double()}
    for e in range(E):
        gu = t["gate_up_weight"][e * 2 * ff:(e + 1) * 2 * ff].double()
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"] = gu[:ff], gu[ff:], t["down_weight"][e * hid:(e + 1) * hid].double()
    mlp = {"router": {"experts": E, "top": top, "scale": scale}}
    if shared:
        w["m.shared.gate"], w["m.shared.up"] = t["shared_gate_up_weight"][:shared].double(), t["shared_gate_up_weight"][shared:].double()
        w["m.shared.down"] = t["shared_down_weight"].double()
        mlp["shared"] = {"ff": shared}
    part.bind({k: (v if k == "correction" else v.to(dt)).to(DEV) for k, v in t.items()})
    h = torch.randn(n, hid, generator=g).to(dt)
    # keep clear of close calls: rows whose choice turns on less than rounding are taken out of the comparison
    s = torch.softmax(h.double() @ w["m.router"].T, -1) + w["m.correction"]
    srt = s.sort(-1, descending=True).values
    clear = torch.ones(n, dtype=torch.bool) if top == E else (srt[:, top - 1] - srt[:, top]) > 1e-5
    ctx = types.SimpleNamespace(n_tokens=n, act_dtype=dt, extras={}, workspace=Workspace(torch.device(DEV)))
    return part, ctx, h, P.experts(h.double(), w, "m.", mlp), clear


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,n,ff,shared,scale", [(5, 2, 150, 24, 40, 1.7), (1, 1, 9, 20, 12, 0.8), (9, 1, 3, 33, 0, 2.0), (3, 3, 70, 64, 9, 1.0),
                                                     (40, 6, 33, 10, 33, 2.5), (16, 4, 1, 40, 24, 1.5), (64, 8, 700, 16, 56, 0.5)])
def test_experts_with_renormalised_weights_and_a_shared_one(dtype, E, top, n, ff, shared, scale):
    """The part on a step's tokens, few (routing in one launch) and many: the correction enters the choice alone, the
    chosen scores are shares of their sum times the factor; the shared expert's inner size may be no multiple of 8."""
    part, ctx, h, want, clear = _expert_case(dtype, E, top, n, ff, shared, scale)
    assert clear.float().mean() > 0.9
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    x0 = torch.randn(n, h.shape[1])
    x = x0.to(DEV).clone()
    part.forward(ctx, h.to(DEV), x, add=True)
    assert rel((x.cpu().double() - x0.double())[clear], want[clear]) < tol
    x = torch.full((n, h.shape[1]), 5.0, device=DEV)
    part.forward(ctx, h.to(DEV), x, add=False)
    assert rel(x[clear.to(DEV)], want[clear]) < tol


@pytest.mark.parametrize("out", ["float32", "bfloat16", None])
@pytest.mark.parametrize("shared,gated", [(0, False), (24, False), (24, True)])
@pytest.mark.parametrize("width,top", [(64, 3), (256, 1), (1032, 6), (2048, 2), (4096, 2)])
def test_norms_around_the_sum_over_experts(out, shared, gated, width, top):
    """Experts' rows by place, weights by pair, a shared row with and without a gate: sum, norm, addition to the stream and
    the next norm in one launch against the same by hand."""
    g = torch.Generator().manual_seed(width + top)
    n, eps, eps2 = 11, 1e-5, 1e-3
    eo, wt = torch.randn(n * top, width, generator=g), torch.rand(n * top, generator=g)
    place = torch.randperm(n * top, generator=g).to(torch.int32)
    sh = torch.randn(n, width, generator=g) if shared else None
    sg = torch.randn(n, 9, generator=g) if gated else None
    x, g1, g2 = torch.randn(n, width, generator=g), 1 + 0.2 * torch.randn(width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    y = (eo.double()[place.long()] * wt.double()[:, None]).view(n, top, width).sum(1)
    if shared:
        y = y + sh.double() * (torch.sigmoid(sg[:, 4].double())[:, None] if gated else 1.0)
    new = x.double() + P.norm(y, g1.double(), eps)
    xs = x.to(DEV).clone()
    nxt = None if out is None else torch.empty(n, width, dtype=DTYPES[out], device=DEV)
    es = K().ExpertSum(eo.to(DEV), wt.to(DEV), place.to(DEV), top, sh.to(DEV) if shared else None, sg.to(DEV)[:, 4] if gated else None)
    K().rmsnorm_add_experts(es, g1.to(DEV), eps, xs, g2.to(DEV) if out else None, eps2, nxt)
    assert rel(xs, new) < 2e-6
    if out is not None:
        assert rel(nxt.float(), P.norm(new, g2.double(), eps2)) < (3e-6 if out == "float32" else 6e-3)
    with pytest.raises(K().KernelError):
        K().rmsnorm_add_experts(es, g1.to(DEV)[:width - 2], eps, xs[:, :width - 2])
    assert not K().rmsnorm_add_experts_fits(4100) and not K().rmsnorm_add_experts_fits(30)


@pytest.mark.parametrize("width,n", [(4, 3), (40, 5), (1024, 7), (2048, 2), (4096, 3), (1000, 33), (4100, 3), (37, 4)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norm_behind_a_sublayer_and_ahead_of_the_next(width, n, dtype):
    """Rows in 16-byte pieces and rows that are not, from a view of a wider matrix too."""
    g = torch.Generator().manual_seed(width)
    y, x = torch.randn(n, width + 8, generator=g), torch.randn(n, width, generator=g)
    g1, g2 = 1 + 0.2 * torch.randn(width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    xs, nxt = x.to(DEV).clone(), torch.empty(n, width, dtype=DTYPES[dtype], device=DEV)
    K().rmsnorm_add_norm(y.to(DEV)[:, 4:4 + width], g1.to(DEV), 1e-5, xs, g2.to(DEV), 1e-4, nxt)
    new = x.double() + P.norm(y[:, 4:4 + width].double(), g1.double(), 1e-5)
    assert rel(xs, new) < 2e-6 and rel(nxt.float(), P.norm(new, g2.double(), 1e-4)) < (3e-6 if dtype == "float32" else 6e-3)


def test_gated_activation_of_float32_projections():
    g = torch.Generator().manual_seed(8)
    for n, f, at in ((5, 16, 16), (130, 1024, 1024), (7, 13, 16), (3, 2056, 2056)):
        gu = torch.randn(n, at + f + 8, generator=g)
        for dt in (torch.float32, torch.bfloat16):
            out = torch.zeros(n, -(-f // 8) * 8, dtype=dt, device=DEV)
            K().gated_act(gu.to(DEV)[:, 4:], out, width=f, up_at=at, gate=K().GATES["silu"])
            want = P.silu(gu[:, 4:4 + f].double()) * gu[:, 4 + at:4 + at + f].double()
            assert rel(out[:, :f].float(), want) < (2e-6 if dt == torch.float32 else 6e-3)


# ---- bounded logits ----------------------------------------------------------------------------------------------

def test_bound_of_the_logits():
    g = torch.Generator().manual_seed(6)
    for shape in ((3, 77), (5, 400), (1, 1), (64, 3001)):
        z = torch.randn(shape, generator=g) * 40
        got = z.to(DEV).clone()
        K().soft_cap(got, 7.5)
        assert rel(got, P.soft_cap(z.double(), 7.5)) < 1e-6
    with pytest.raises(K().KernelError):
        K().soft_cap(got, 0.0)


@pytest.mark.parametrize("rows,vocab,k", [(8, 50257, 64), (3, 301, 136), (40, 50257, 64), (100, 33000, 64)])
def test_tokens_chosen_in_the_product_from_bounded_logits(rows, vocab, k):
    """The three kernels with the epilogue: rows with a temperature draw what the sampling kernel draws from the bounded
    logits (for logits far beyond the bound that is another token than without it), the others take the arg-max."""
    g = torch.Generator().manual_seed(rows)
    a = torch.randn(rows, k, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(vocab, k, generator=g)).to(torch.bfloat16).to(DEV)
    logits, cap = torch.empty(rows, vocab, device=DEV), 2.0
    K().linear(a, w, None, logits, path=K().bf16_path(rows, vocab, k, out_f32=True))
    top = logits.argmax(1).tolist()
    temps = torch.tensor([0.0, 0.7, 1.0, 1.3, 0.8, 2.0, 0.0, 0.5] * 20)[:rows].to(DEV)
    seeds, want, got, free = (torch.arange(rows, dtype=torch.int64) * 7919).to(DEV), *(torch.empty(rows, dtype=torch.int32, device=DEV) for _ in range(3))
    bounded = logits.clone()
    K().soft_cap(bounded, cap)
    differs = 0
    for step in range(4):
        counters = (torch.arange(rows, dtype=torch.int32) + step).to(DEV)
        K().sample(bounded, temps, None, None, seeds, counters, want)
        K().linear_sample(a, w, None, K().SampleInto(got, temps, seeds, counters), soft_cap=cap)
        K().linear_sample(a, w, None, K().SampleInto(free, temps, seeds, counters))
        for r in range(rows):
            assert int(got[r]) == (int(want[r]) if float(temps[r]) > 0 else top[r])
        differs += int((got != free).sum())
    assert differs > 0
    K().linear_sample(a, w, None, K().SampleInto(got), soft_cap=cap)
    assert got.tolist() == top


# ---- whole models through the step function ------------------------------------------------------------

@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("kugadra"))
    return {(name, dtype): write_tiny(name, root, decisive=dtype == "bfloat16") for name in TINY for dtype in DTYPES}


_plain: dict = {}


def plain_logits(folder, toks, how="exact"):
    """``exact``: float64.  ``float32``: the same functions on float32 tensors.  ``bfloat16``: float64 with the
    activations rounded to bfloat16 where a 16-bit engine stores them.  The last two show how far rounding alone
    moves the logits of this very sequence, which is what the tolerances below are tied to."""
    key = (folder, tuple(toks), how)
    if key not in _plain:
        if folder not in _plain:
            cfg, w = load_folder(folder)
            _plain[folder] = (cfg, w, {k: v.float() for k, v in w.items()})
        cfg, w, w32 = _plain[folder]
        if how == "float32":
            _plain[key] = P.forward(cfg, w32, toks).double()
        else:
            _plain[key] = P.forward(cfg, w, toks, rounding=P.to_bfloat16_and_back if how == "bfloat16" else None)
    return _plain[key]


def centred_rms(d):
    d = d - d.mean()
    return float(d.pow(2).mean().sqrt())


def row_limit(folder, toks, pos, dtype):
    """float32: 3e-4 on a logit, or five times what float32 rounding moves this row in the plain implementation.
    bfloat16: the row's error (mean taken off, root mean square over the vocabulary, over that of the plain row) 0.08, or
    three times what bfloat16 storage moves it."""
    ref = plain_logits(folder, toks)[pos]
    if dtype == "float32":
        return max(3e-4, 5.0 * float((plain_logits(folder, toks, "float32")[pos] - ref).abs().max()))
    return max(0.08, 3.0 * centred_rms(plain_logits(folder, toks, "bfloat16")[pos] - ref) / centred_rms(ref))


def check(folder, reqs, trace, got, dtype):
    """Every wanted row within ``row_limit`` of the plain logits: in float32 all rows, in bfloat16 all but 2 %."""
    over, total, errs = 0, 0, []
    for s, want in zip(trace.steps, trace.wanted):
        if not want:
            continue
        arr = torch.from_numpy(got[s["step"]].astype(np.float64)).view(len(want), -1)
        for row, (rid, pos) in enumerate(want):
            ref = plain_logits(folder, reqs[rid])[pos]
            assert torch.isfinite(arr[row]).all()
            total += 1
            limit = row_limit(folder, reqs[rid], pos, dtype)
            if dtype == "float32":
                diff = float((arr[row] - ref).abs().max())
                assert diff <= limit, (f"step {s['step']}: request {rid} position {pos}: |logits - plain| = {diff:.3e} > "
                                       f"{limit:.1e}; entries {[(e['id'], len(e['tokens'])) for e in s['entries']]}")
            else:
                errs.append(centred_rms(arr[row] - ref) / centred_rms(ref))
                over += errs[-1] > limit
    assert over <= 0.02 * total + 1, (f"{over} of {total} rows differ from the plain logits beyond bfloat16 rounding; "
                                      f"quantiles 50/90/99 %: {np.quantile(errs, [0.5, 0.9, 0.99])}")


def requests_for(name, lens, seed):
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, TINY[name]["raw"]["vocab"], size=n).tolist() for i, n in enumerate(lens)}


def replay(folder, name, dtype, trace, out, **kw):
    return R.replay(folder, dtype, trace, str(out), page_size=TINY[name]["page_size"], **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_whole_prompts(folders, tmp_path, name, dtype):
    f = folders[name, dtype]
    reqs = requests_for(name, [1, 2, 5, 16, 17, 63, 65, 150, 300], 1)
    tr = R.whole(reqs)
    check(f, reqs, tr, replay(f, name, dtype, tr, tmp_path), dtype)


def test_every_layer_against_the_plain_stream(folders):
    """The stream after each layer, in 32 bits."""
    from rosellm_b200.config.engine import EngineConfig
    from rosellm_b200.engine.runner import ModelRunner, StepEntry

    for name in TINY:
        f = folders[name, "float32"]
        runner = ModelRunner.from_folder(f, EngineConfig(dtype="float32", page_size=TINY[name]["page_size"], kv_cache_tokens=256,
                                                         max_num_seqs=2, cuda_graphs=False, capture_graphs_at_start=False, device=DEV))
        caught = []
        for layer in runner.model.layers:
            def wrapped(ctx, run, lyr, x, inner=layer.block.forward):
                inner(ctx, run, lyr, x)
                caught.append(x.detach().cpu().clone())
            layer.block.forward = wrapped
        toks = requests_for(name, [70], 11)["r0"]
        slot = runner.cache.new_request()
        runner.step([StepEntry(slot, toks, [len(toks) - 1])])
        runner.check_status()
        cfg, w = load_folder(f)
        streams = []
        P.forward(cfg, w, toks, streams=streams)
        assert len(caught) == len(streams) == len(cfg["layers"])
        for i, (mine, want) in enumerate(zip(caught, streams)):
            assert rel(mine, want) < 3e-5, (name, i)


@pytest.mark.parametrize("graphs", [False, True], ids=["walked", "graphs"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_prefill_against_token_by_token_decoding(folders, tmp_path, name, dtype, graphs):
    """The last 40 tokens one by one (with ``graphs``: as CUDA-graph replays, the way generation runs them), over
    page and chunk borders."""
    f = folders[name, dtype]
    reqs = requests_for(name, [41, 72, 104, 3], 2)
    tr = R.tail_decoded(reqs, tail=40)
    stats = {}
    got = replay(f, name, dtype, tr, tmp_path, cuda_graphs=graphs, stats=stats)
    check(f, reqs, tr, got, dtype)
    assert (stats["graph_replays"] > 0) == graphs


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_portions_down_to_two_tokens(folders, tmp_path, name, dtype):
    f = folders[name, dtype]
    reqs = requests_for(name, [100, 37, 64, 129], 3)
    for sizes in ((7, 2, 16, 3, 2, 5, 33, 2, 1, 17), (2,), (15, 1, 16, 17), (64, 63, 2)):
        tr = R.portions(reqs, sizes=sizes)
        got = replay(f, name, dtype, tr, tmp_path / f"s{len(sizes)}{sizes[0]}")
        check(f, reqs, tr, got, dtype)


@pytest.mark.parametrize("graphs", [False, True], ids=["walked", "graphs"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_mixed_batches_with_pages_and_slots_used_again(folders, tmp_path, name, dtype, graphs):
    """Up to four live requests, portions beside single tokens, in a pool so small that pages and slots come
    round again; every row is compared with the request run alone (the plain implementation knows no batch): a
    key left over by a page's earlier owner, or a state by a slot's, would show."""
    f = folders[name, dtype]
    lens = [120, 9, 200, 33, 70, 2, 193, 64, 20, 101]
    reqs = requests_for(name, lens, 4)
    prompt_lens = {rid: max(1, len(t) - (8 if i % 2 else 40)) for i, (rid, t) in enumerate(reqs.items())}
    tr = R.mixed(reqs, prompt_lens, max_live=4, seed=5)
    peak = R.peak_tokens(tr)
    assert sum(-(-len(t) // 64) * 64 for t in reqs.values()) > 1.5 * peak
    got = replay(f, name, dtype, tr, tmp_path, max_tokens=peak, cuda_graphs=graphs)
    check(f, reqs, tr, got, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(folders, tmp_path, dtype):
    f = folders["A", dtype]
    reqs = requests_for("A", [1, 2, 3, 4], 9)
    for i, tr in enumerate((R.whole(reqs), R.tail_decoded(reqs, tail=10), R.portions(reqs, sizes=(2, 1)))):
        check(f, reqs, tr, replay(f, "A", dtype, tr, tmp_path / f"f{i}"), dtype)
    for name in ("B", "F"):
        f = folders[name, dtype]
        reqs = requests_for(name, [420], 10)
        tr = R.tail_decoded(reqs, tail=417)
        check(f, reqs, tr, replay(f, name, dtype, tr, tmp_path / f"long{name}", cuda_graphs=True), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wide_model_with_long_contexts(tmp_path, dtype):
    """Width 1024: the products' tensor-core paths with float32 outputs, prompts of 600 and 350 tokens whole and in
    portions of up to 256, the last tokens one by one, ten chunks of the linear attention, a latent of 256."""
    folder = write_tiny("WIDE", str(tmp_path), decisive=dtype == "bfloat16")
    rng = np.random.default_rng(3)
    reqs = {f"r{i}": rng.integers(0, WIDE["raw"]["vocab"], size=n).tolist() for i, n in enumerate([600, 350])}
    for i, tr in enumerate((R.whole(reqs), R.tail_decoded(reqs, tail=6), R.portions(reqs, sizes=(256, 3, 130, 64, 200)))):
        wanted = {rid: {len(t) - 1, len(t) - 2, len(t) // 2, 0, 1} for rid, t in reqs.items()}
        for s_, w_ in zip(tr.steps, tr.wanted):  # keep a few rows a request: the logits of 950 rows are not needed
            keep = [k for k, (rid, pos) in enumerate(w_) if pos in wanted[rid] or len(s_["entries"][0]["tokens"]) == 1]
            at = 0
            for e in s_["entries"]:
                n = len(e["want"])
                e["want"] = [e["want"][k - at] for k in keep if at <= k < at + n]
                at += n
            w_[:] = [w_[k] for k in keep]
        got = R.replay(folder, dtype, tr, str(tmp_path / f"w{i}"), page_size=16)
        check(folder, reqs, tr, got, dtype)


def test_trace_program_as_a_child_process(folders, tmp_path):
    f = folders["A", "float32"]
    reqs = requests_for("A", [40, 90, 3], 6)
    tr = R.mixed(reqs, {rid: len(t) - 5 for rid, t in reqs.items()}, max_live=2, seed=1)
    got = R.replay(f, "float32", tr, str(tmp_path), subprocess_mode=True, page_size=16)
    check(f, reqs, tr, got, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    """Prompts of unequal length through ``InferenceEngine.generate_batch`` (scheduler, portions of 16 tokens,
    decode graphs, tokens chosen on the device and fed back without the host reading them): every generated token is the
    plain arg-max given the tokens before it, or within the precision's reach."""
    from rosellm_b200.engine.llm import InferenceEngine

    f = folders[name, dtype]
    rng = np.random.default_rng(7)
    vocab = TINY[name]["raw"]["vocab"]
    prompts = [rng.integers(0, vocab, n).tolist() for n in (5, 37, 1, 64)]
    eng = InferenceEngine(f, dtype=dtype, page_size=TINY[name]["page_size"], max_batch_size=4,
                          kv_cache_max_tokens=512, prefill_chunk_size=16, max_position_embeddings=256)
    outs = eng.generate_batch(prompts, max_new_tokens=12, stop_on_eos=False)
    assert [len(o) for o in outs] == [12] * 4
    for prompt, out in zip(prompts, outs):
        ids = list(prompt)
        for tok in out:
            ref = plain_logits(f, ids)[-1]
            gap = float(ref.max() - ref[tok])
            limit = row_limit(f, ids, len(ids) - 1, dtype)  # on a logit, or on the row's relative error
            assert gap <= (2 * limit if dtype == "float32" else 1.4 * limit * centred_rms(ref)), (gap, limit)
            ids.append(tok)


def test_sampling_with_a_temperature_uses_bounded_logits(folders):
    """Generation with a temperature, tokens chosen in the head's product and from written logits: the same tokens, and
    tokens that the bounded plain logits explain."""
    from rosellm_b200.engine.llm import InferenceEngine

    f = folders["A", "bfloat16"]
    prompts = [[5, 17, 3], [99, 1, 2, 3, 4, 5, 6]]
    outs = []
    for in_head in (True, False):
        eng = InferenceEngine(f, dtype="bfloat16", page_size=16, max_batch_size=2, kv_cache_max_tokens=512, prefill_chunk_size=16,
                              max_position_embeddings=256)
        eng.sample_in_head = in_head
        outs.append(eng.generate_batch(prompts, max_new_tokens=60, stop_on_eos=False, temperature=0.9, do_sample=True, seed=3))
    assert outs[0] == outs[1] and [len(o) for o in outs[0]] == [60, 60]
    for prompt, out in zip(prompts, outs[0]):
        ids, gaps = list(prompt), []
        for tok in out:
            ref = plain_logits(f, ids)[-1]
            gaps.append(float(ref.max() - ref[tok]) / 0.9)
            ids.append(tok)
        # draws from 131 entries whose logits lie within 2 x 2.5: a gap beyond what the bound leaves has no chance
        assert max(gaps) < 5.0 / 0.9 + 0.2 and len(set(out)) > 20


def test_preemption_changes_no_token(folders):
    """A pool too small for four requests at once: the one admitted last gives its pages and its state back and is
    recomputed; the tokens are those of a run with room for all."""
    from rosellm_b200.engine.llm import InferenceEngine

    f = folders["F", "float32"]
    rng = np.random.default_rng(8)
    prompts = [rng.integers(0, 64, n).tolist() for n in (30, 25, 40, 20)]
    outs = []
    for tokens in (512, 160):
        eng = InferenceEngine(f, dtype="float32", page_size=8, max_batch_size=4, kv_cache_max_tokens=tokens, prefill_chunk_size=16,
                              max_position_embeddings=128)
        outs.append(eng.generate_batch(prompts, max_new_tokens=40, stop_on_eos=False))
        assert (eng.num_preemptions > 0) == (tokens == 160)
    assert outs[0] == outs[1] and [len(o) for o in outs[0]] == [40] * 4


def test_the_command_line_generates_the_plain_greedy_tokens(folders):
    """``python -m rosellm_b200.cli_generate`` as a child process, in 32 bits: the ids it prints are the plain arg-max,
    token after token."""
    import ast
    import subprocess
    import sys

    f = folders["A", "float32"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    prompt = np.random.default_rng(12).integers(0, TINY["A"]["raw"]["vocab"], 23).tolist()
    env = dict(os.environ, PYTHONPATH=root + os.pathsep + os.environ.get("PYTHONPATH", ""))
    res = subprocess.run([sys.executable, "-m", "rosellm_b200.cli_generate", "--model", f, "--prompt-ids",
                          ",".join(map(str, prompt)), "--max-new-tokens", "6", "--no-stop-on-eos", "--dtype", "fp32",
                          "--max-num-batched-tokens", "64", "--max-num-seqs", "2", "--page-size", str(TINY["A"]["page_size"]),
                          "--kv-cache-max-tokens", "256"],
                         capture_output=True, text=True, timeout=600, env=env, cwd=root)
    assert res.returncode == 0, res.stderr[-3000:]
    line = next(l for l in res.stdout.splitlines() if l.startswith("[rosellm_b200] output: "))
    got = list(ast.literal_eval(line.split(": ", 1)[1]))
    assert len(got) == 6
    ids = list(prompt)
    for tok in got:
        ref = plain_logits(f, ids)[-1]
        assert float(ref.max() - ref[tok]) <= 2 * row_limit(f, ids, len(ids) - 1, "float32")
        ids.append(tok)

"""Vebotar on the GPU: every mechanism's kernels against the plain implementation's function for it, then whole
models through the engine's step function, cache, scheduler and entry point."""
import os
import types

import numpy as np
import pytest
import torch

import plain_vebotar as P
import replay_util as R
from tiny_vebotar import TINY, WIDE, load_folder, write_tiny

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


# ---- the stream's copies ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("copies", [1, 2, 3, 4, 5, 8, 11, 16])
@pytest.mark.parametrize("width", [24, 101, 1000, 4096])
def test_reading_and_writing_the_copies(dtype, copies, width):
    """The first read (one row for all copies), a write from that row, writes in place, the last write into the sum;
    widths with and without 16-byte rows; one to sixteen copies; weights of both signs."""
    g = torch.Generator().manual_seed(copies * width)
    n, eps, dt = 5, 1e-3, DTYPES[dtype]
    r = lambda *s: torch.randn(*s, generator=g)
    a, b, M, a2, gamma, gamma2 = r(copies), r(copies), r(copies, copies) / copies ** 0.5, r(copies), r(width), r(width)
    x0, y, y2 = r(n, width), r(n, width), r(n, width)
    D = lambda t: t.double()
    tol = 3e-6 if dtype == "float32" else 6e-3

    def normed(X, w, gm):
        return P.unit(P.read_streams(X, D(w)), eps) * D(gm)

    X = D(x0)[None].repeat(copies, 1, 1)
    xd, h = x0.to(DEV), torch.empty(n, width, dtype=dt, device=DEV)
    K().hyper_step(xd, None, copies=copies, read=a.to(DEV), gamma=gamma.to(DEV), eps=eps, h=h)
    if float(a.sum().abs()) > 0.05:  # weights that nearly cancel leave a sum that rounding alone makes
        assert rel(h.float(), normed(X, a, gamma)) < 30 * tol
    Xd = torch.full((n, copies, width), 9.0, device=DEV)
    K().hyper_step(xd, y.to(DEV), copies=copies, write=(M.to(DEV), b.to(DEV)), x_new=Xd, read=a2.to(DEV), gamma=gamma2.to(DEV),
                   eps=eps, h=h)
    X = P.write_streams(X, D(M), D(b), D(y))
    assert rel(Xd.transpose(0, 1), X) < 3e-6 and rel(h.float(), normed(X, a2, gamma2)) < tol
    assert torch.equal(xd.cpu(), x0)
    K().hyper_step(Xd, y2.to(DEV), copies=copies, write=(M.to(DEV), b.to(DEV)), x_new=Xd, read=a.to(DEV), gamma=gamma.to(DEV),
                   eps=eps, h=h)  # in place
    X = P.write_streams(X, D(M), D(b), D(y2))
    assert rel(Xd.transpose(0, 1), X) < 5e-6 and rel(h.float(), normed(X, a, gamma)) < 10 * tol
    total = torch.empty(n, width, device=DEV)
    K().hyper_step(Xd, y.to(DEV), copies=copies, write=(M.to(DEV), b.to(DEV)), total=total)
    assert rel(total, P.write_streams(X, D(M), D(b), D(y)).sum(0)) < 2e-5
    K().hyper_step(xd, y.to(DEV), copies=copies, write=(M.to(DEV), b.to(DEV)), total=xd)  # a model of one sublayer: into its own row
    assert rel(xd, P.write_streams(D(x0)[None].repeat(copies, 1, 1), D(M), D(b), D(y)).sum(0)) < 2e-5


@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("width,top", [(64, 3), (30, 1), (520, 6)])
def test_writing_the_copies_from_unsummed_experts(width, top, shared):
    g = torch.Generator().manual_seed(width)
    n, copies = 9, 3
    eo = torch.randn(n * top, width, generator=g)
    place = torch.randperm(n * top, generator=g).to(torch.int32)
    weights = torch.rand(n * top, generator=g)
    sh, z = torch.randn(n, width, generator=g), torch.randn(n, 8, generator=g) * 3.0
    y = (eo[place.long()].double().view(n, top, width) * weights.double().view(n, top, 1)).sum(1)
    if shared:
        y = y + torch.sigmoid(z[:, 5:6].double()) * sh.double()
    X, M, b = torch.randn(n, copies, width, generator=g), torch.randn(copies, copies, generator=g), torch.randn(copies, generator=g)
    zd = z.to(DEV)
    s = K().ExpertSum(eo.to(DEV), weights.to(DEV), place.to(DEV), top, sh.to(DEV) if shared else None, zd[:, 5] if shared else None)
    Xd = X.to(DEV)
    total = torch.empty(n, width, device=DEV)
    K().hyper_step(Xd, s, copies=copies, write=(M.to(DEV), b.to(DEV)), x_new=Xd, total=total)
    want = P.write_streams(X.double().transpose(0, 1), M.double(), b.double(), y)
    assert rel(Xd.transpose(0, 1), want) < 3e-6 and rel(total, want.sum(0)) < 1e-5


def test_refused_copies():
    x = torch.zeros(2, 17, 8, device=DEV)
    w, m = torch.zeros(17, device=DEV), torch.zeros(17, 17, device=DEV)
    with pytest.raises(K().KernelError):
        K().hyper_step(x, torch.zeros(2, 8, device=DEV), copies=17, write=(m, w), x_new=x, total=torch.zeros(2, 8, device=DEV))
    with pytest.raises(K().KernelError):
        K().hyper_step(x[:, :2].contiguous(), None, copies=2)


# ---- experts -----------------------------------------------------------------------------------------

@pytest.mark.parametrize("experts,top,n", [(5, 2, 150), (1, 1, 9), (9, 1, 3), (3, 3, 70), (40, 6, 128), (40, 40, 33), (256, 8, 2), (64, 4, 700)])
def test_routing_by_the_chosen_logits(experts, top, n):
    """The largest logits, weighted by the softmax over them alone, whatever the other logits are; in one launch with the
    layout (few tokens) and in three; logits that are columns of a wider matrix."""
    g = torch.Generator().manual_seed(experts + n)
    z = torch.randn(n, experts + 3, generator=g) * 4.0
    zd = z.to(DEV)[:, :experts]
    idx, weight = P.route(z[:, :experts].double(), top)
    i32 = lambda m: torch.full((m,), -7, dtype=torch.int32, device=DEV)
    choice = dict(top=top, group_count=1, group_keep=1, score=K().MOE_SCORES["chosen_softmax"])
    for fused in ((False, True) if n <= K().MOE_ROUTE_MAX_TOKENS else (False,)):
        ids, w = i32(n * top), torch.zeros(n * top, device=DEV)
        offsets, tiles, meta = i32(experts + 1), i32(3 * K().moe_max_tiles(n * top, experts)), i32(4)
        row_token, place = i32(n * top), i32(n * top)
        if fused:
            K().moe_select_route(zd, None, ids=ids, weights=w, offsets=offsets, tiles=tiles, meta=meta, row_token=row_token,
                                 place_of=place, **choice)
        else:
            counts, fill = torch.zeros(experts, dtype=torch.int32, device=DEV), torch.zeros(experts, dtype=torch.int32, device=DEV)
            K().moe_select(zd, None, ids=ids, weights=w, counts=counts, **choice)
            K().moe_plan(ids, counts, fill, offsets, tiles, meta, row_token, place, n_tokens=n, n_experts=experts, top=top)
            assert not counts.any()
        assert torch.equal(ids.view(n, top).cpu().long(), idx) and rel(w.view(n, top), weight) < 2e-6
        off = offsets.cpu().tolist()
        per = torch.bincount(idx.flatten(), minlength=experts).tolist()
        assert [off[e + 1] - off[e] for e in range(experts)] == per
        p = place.cpu().tolist()
        assert sorted(p) == list(range(n * top))
        for pair, at in enumerate(p):
            e = int(idx.flatten()[pair])
            assert off[e] <= at < off[e + 1] and int(row_token[at]) == pair // top
        t = tiles.cpu().view(-1, 3)[:int(meta[0])].tolist()
        assert sum(r for _, _, r in t) == n * top and all(0 < r <= 64 and off[e] <= a and a + r <= off[e + 1] for e, a, r in t)


@pytest.mark.parametrize("score", ["softmax", "sigmoid", "chosen_softmax"])
def test_routing_in_one_launch_equals_routing_in_three(score):
    """Also with a correction of the choice, groups, and weights left by place (what other designs ask of it)."""
    g = torch.Generator().manual_seed(4)
    n, E, top = 100, 24, 5
    z, corr = (torch.randn(n, E, generator=g) * 3.0).to(DEV), torch.randn(E, generator=g).to(DEV)
    i32 = lambda m: torch.zeros(m, dtype=torch.int32, device=DEV)
    for correction, groups, keep in ((None, 1, 1), (corr, 1, 1), (None, 6, 3), (corr, 4, 2)):
        choice = dict(top=top, group_count=groups, group_keep=keep, score=K().MOE_SCORES[score])
        res = []
        for fused in (False, True):
            ids, w, pw = i32(n * top), torch.zeros(n * top, device=DEV), torch.zeros(n * top, device=DEV)
            offsets, tiles, meta, row_token, place = i32(E + 1), i32(3 * K().moe_max_tiles(n * top, E)), i32(4), i32(n * top), i32(n * top)
            if fused:
                K().moe_select_route(z, correction, ids=ids, weights=w, offsets=offsets, tiles=tiles, meta=meta,
                                     row_token=row_token, place_of=place, place_weight=pw, **choice)
            else:
                counts, fill = i32(E), i32(E)
                K().moe_select(z, correction, ids=ids, weights=w, counts=counts, **choice)
                K().moe_plan(ids, counts, fill, offsets, tiles, meta, row_token, place, n_tokens=n, n_experts=E, top=top,
                             weights=w, place_weight=pw)
            m = int(meta[0])
            res.append((ids, w, offsets, tiles[:3 * m], pw[place.long()], row_token[place.long()]))
        for a, b in zip(*res):
            assert torch.equal(a, b)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,n,ff,shared", [(5, 2, 150, 24, 40), (1, 1, 9, 20, 12), (9, 1, 3, 33, 0), (3, 3, 70, 64, 9),
                                                     (16, 4, 1, 48, 72), (8, 2, 600, 100, 0), (40, 6, 200, 10, 130)])
def test_experts_of_one_projection_and_the_shared_expert(dtype, experts, top, n, ff, shared):
    """The part itself: few tokens (every expert's weights streamed once) and many (tiles), inner sizes that are no
    multiple of 8, with and without a shared expert; summed, added, and left unsummed for the stream's kernel."""
    from rosellm_b200.engine.context import Workspace
    from rosellm_b200.parts.gated import MixtureOfExperts

    g = torch.Generator().manual_seed(experts * 7 + top)
    dt, hid = DTYPES[dtype], 48
    part = MixtureOfExperts(hidden_size=hid, inner_size=ff, num_experts=experts, top=top, gate="relu_squared",
                            score="chosen_softmax", shared_inner=shared)
    r = lambda *s: (torch.randn(*s, generator=g) * 0.3).to(torch.bfloat16)
    up, down, router = r(experts * ff, hid), r(experts * hid, ff), r(experts, hid)
    t = {"up_weight": up, "down_weight": down, "router_weight": router}
    w = {"m.router": router.double()}
    for e in range(experts):
        w[f"m.e{e}.up"], w[f"m.e{e}.down"] = up[e * ff:(e + 1) * ff].double(), down[e * hid:(e + 1) * hid].double()
    mlp = {"router": {"experts": experts, "top": top}}
    if shared:
        t.update(shared_up_weight=r(shared, hid), shared_down_weight=r(hid, shared), shared_gate_weight=r(1, hid) * 4)
        w.update({"m.shared.up": t["shared_up_weight"].double(), "m.shared.down": t["shared_down_weight"].double(),
                  "m.shared.sg": t["shared_gate_weight"].double()})
        mlp["shared"] = {"ff": shared}
    assert {s.role for s in part.param_specs()} == set(t)
    part.bind({k: v.to(dt).to(DEV) for k, v in t.items()})
    h = torch.randn(n, hid, generator=g).to(dt)
    z = h.double() @ w["m.router"].T
    want = P.experts(h.double(), w, "m.", mlp)
    if experts > top:  # leave out tokens whose choice is a close call
        v = z.sort(-1, descending=True).values
        keep = (v[:, top - 1] - v[:, top]) > 1e-3
    else:
        keep = torch.ones(n, dtype=torch.bool)
    ctx = types.SimpleNamespace(n_tokens=n, act_dtype=dt, extras={}, workspace=Workspace(torch.device(DEV)))
    x0 = torch.randn(n, hid, generator=g)
    x = x0.to(DEV).clone()
    part.forward(ctx, h.to(DEV), x, add=True)
    K().check_status(torch.device(DEV))
    tol = 2e-5 if dtype == "float32" else 1.5e-2
    assert rel((x.cpu().double() - x0.double())[keep], want[keep]) < tol
    part.forward(ctx, h.to(DEV), x, add=False)
    assert rel(x.cpu()[keep], want[keep]) < tol
    left = part.forward_deferred(ctx, h.to(DEV))
    total = torch.empty(n, hid, device=DEV)
    one = torch.ones(1, device=DEV)
    K().hyper_step(torch.zeros(n, hid, device=DEV), left, copies=1, write=(one, one), total=total)
    assert rel(total.cpu()[keep], want[keep]) < tol


@pytest.mark.parametrize("rows", [1, 7, 16, 40, 64, 100, 128, 300])
def test_squared_relu_behind_a_product(rows):
    """Every matrix kernel's epilogue."""
    g = torch.Generator().manual_seed(rows)
    for dt, n_out, k in ((torch.bfloat16, 136, 256), (torch.bfloat16, 1024, 1024), (torch.bfloat16, 2056, 64), (torch.float32, 72, 96)):
        a, w, b = torch.randn(rows, k, generator=g).to(dt), (torch.randn(n_out, k, generator=g) * k ** -0.5).to(dt), torch.randn(n_out, generator=g)
        for bias in (None, b):
            out = torch.empty(rows, n_out, dtype=dt, device=DEV)
            K().linear(a.to(DEV), w.to(DEV), None if bias is None else bias.to(DEV), out, act=K().ACT_RELU_SQUARED)
            want = torch.clamp(a.double() @ w.double().T + (0.0 if bias is None else bias.double()), min=0.0) ** 2
            assert rel(out.float(), want) < (1e-5 if dt == torch.float32 else 8e-3), (dt, n_out, k)


# ---- queries, keys and values ahead of the cache -------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,rot", [(6, 2, 20, 12, 12), (4, 4, 64, 32, 64), (7, 1, 9, 5, 8), (2, 1, 136, 130, 20)])
def test_turning_two_maps_and_filling_the_cache(dtype, H, G, dk, dv, rot):
    """Both vectors of a head turned alike with scaled cosines, entries beyond the turned ones untouched; a cache row is
    [key 1 | key 2 | value]; a padding row writes nothing; queries alone when the layer reads another's cache."""
    from rosellm_b200.engine.context import build_host_batch
    from rosellm_b200.parts.standard import RotaryPositions

    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(H + dk)
    page, v_at = 8, -(-2 * dk // 8) * 8
    row = -(-(v_at + dv) // 8) * 8
    hb = build_host_batch([(1, 5, [0] * 20, []), (2, 0, [0] * 3, []), (3, 31, [0], []), (-1, 0, [0], [])])
    n = len(hb.positions)
    table = torch.full((4, 8), -1, dtype=torch.int32)
    table[1:, :] = torch.randperm(24, generator=g).view(3, 8).to(torch.int32)
    q, k, v = (torch.randn(n, w, generator=g) for w in (H * 2 * dk, G * 2 * dk, G * dv))
    sc = dict(factor=6.0, original=16, fast=4.0, slow=0.5)
    rp = RotaryPositions(dims=rot, base=300.0, scaling=dict(sc, kind="ramp"))
    freqs, mult = P.ramp_frequencies(rot, 300.0, sc)
    assert mult > 1.15
    pool = torch.full((24, 1, G, page, row), 7.0, dtype=dt, device=DEV)
    bq, bk, bv = q.to(DEV).clone(), k.to(DEV).clone(), v.to(DEV).clone()
    common = dict(n_heads=H, n_kv=G, dk=dk, dv=dv, eps=1e-5, freq=rp.frequencies(DEV), rot_dims=rot, maps=2, rot_mult=rp.mult)
    K().qkv_norm_rotate(bq, bk, bv, dev(hb.positions), cache=K().QkvCache(pool, table.to(DEV), dev(hb.req_of_token), dev(hb.slots), v_at, 64),
                        **common)
    K().check_status(torch.device(DEV))
    pos = torch.from_numpy(hb.positions)
    want_q = P.turn(q.double().view(n, H, 2, dk), pos, freqs, mult)
    want_k = P.turn(k.double().view(n, G, 2, dk), pos, freqs, mult)
    assert rel(bq.view(n, H, 2, dk), want_q) < 2e-5
    alone = q.to(DEV).clone()
    K().qkv_norm_rotate(alone, None, None, dev(hb.positions), **common)
    assert torch.equal(alone, bq)
    tol = 2e-5 if dtype == "float32" else 5e-3
    for t in range(n - 1):
        slot, p = int(hb.slots[hb.req_of_token[t]]), int(pos[t])
        r = pool[int(table[slot, p // page]), 0, :, p % page].float().cpu()
        assert rel(r[:, :2 * dk].reshape(G, 2, dk), want_k[t]) < tol and rel(r[:, v_at:v_at + dv], v[t].view(G, dv)) < tol
    assert (pool != 7.0).sum() == (n - 1) * G * (2 * dk + dv)


# ---- attention ------------------------------------------------------------------------------------------

def one_map(q, k, v, scale, size):
    """A single softmax map by the plain function for two: the first of two equal maps."""
    return P.two_maps(q[:, :, None].expand(-1, -1, 2, -1), k[:, :, None].expand(-1, -1, 2, -1), v, scale, size)[:, :, 0]


def _attn_case(dtype, H, G, dk, dv, lens_new, lens_old, page, scale, chunk, seed, *, maps=2, lam=0.7, diff=0.3, eps=1e-3,
               stand_out=None, splits=1, mma=False):
    """Requests with ``lens_old`` cached tokens bring ``lens_new`` more.  All tokens' cache rows are written by the
    store kernel; then the pages of chunks that the sequence has left before this step are taken away (their table
    entries -1, their rows overwritten with huge numbers), as the cache manager does.  Returns the kernel's output
    [tokens, H, dv], the plain result from the same (rounded) keys and values, the values, and the two plain maps."""
    from rosellm_b200.engine.context import build_host_batch

    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(seed)
    v_at = -(-maps * dk // 8) * 8
    row = -(-(v_at + dv) // 8) * 8
    n_req = len(lens_new)
    totals = [a + b for a, b in zip(lens_new, lens_old)]
    pages_per = [-(-t // page) for t in totals]
    n_pages = sum(pages_per) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((n_req + 1, max(pages_per)), -1, dtype=torch.int32)
    at = 0
    for r in range(n_req):
        for lp in range(pages_per[r]):
            table[r + 1, lp] = order[at]
            at += 1
    pool = torch.full((n_pages, 1, G, page, row), 9.0, dtype=dt, device=DEV)
    ks = [torch.randn(t, G, maps, dk, generator=g) * 0.7 for t in totals]
    vs = [torch.randn(t, G, dv, generator=g) for t in totals]
    n_tok = sum(lens_new)
    q = torch.randn(n_tok, H, maps, dk, generator=g) * 0.8
    if stand_out is not None:  # request 0's last query points hard at one key, in one map
        key, head, m = stand_out
        ks[0][key, head // (H // G), m] = q[lens_new[0] - 1, head, m] * 40.0
    full = table.to(DEV)
    for new, old in ((lens_old, [0] * n_req), (lens_new, lens_old)):
        ents = [(r + 1, old[r], [0] * new[r], []) for r in range(n_req) if new[r] > 0]
        if not ents:
            continue
        hb = build_host_batch(ents)
        kk = torch.cat([ks[r][old[r]:old[r] + new[r]] for r in range(n_req) if new[r] > 0]).reshape(-1, G * maps * dk)
        vv = torch.cat([vs[r][old[r]:old[r] + new[r]] for r in range(n_req) if new[r] > 0]).reshape(-1, G * dv)
        K().bias_kv_store(kk.to(DEV), vv.to(DEV), pool, full, dev(hb.positions), dev(hb.req_of_token), dev(hb.slots),
                          v_at=v_at, max_pos=max(totals))
    if chunk is not None:
        for r in range(n_req):
            for lp in range(lens_old[r] // chunk * chunk // page):
                pool[int(table[r + 1, lp])] = 1e4
                table[r + 1, lp] = -1
    table = table.to(DEV)
    mma = mma and K().bias_attention_tensor_cores(dt, dk, dv, maps)
    wide = K().bias_attention_shape(H // G, mma, maps)[1] > 16
    tiles, n_tiles = (hb.tiles_wide, len(hb.tiles_wide)) if wide else (hb.tiles, len(hb.tiles))
    out = torch.full((n_tok, H * dv), 5.0, dtype=dt, device=DEV)
    part_o = part_ml = None
    if splits > 1:
        part_o = torch.full((len(hb.decode_reqs) * H * maps * splits, dv), float("nan"), device=DEV)
        part_ml = torch.full((len(hb.decode_reqs) * H * maps * splits, 2), float("nan"), device=DEV)
    two = dict(maps=2, diff_lambda=torch.tensor([lam], device=DEV), diff_eps=eps, diff_mul=1.0 - diff) if maps == 2 else {}
    K().bias_attention(q.reshape(n_tok, H * maps * dk).to(DEV), None, pool, table, dev(hb.q_start), dev(hb.kv_len), dev(hb.slots), out,
                       n_heads=H, dk=dk, dv=dv, v_at=v_at, scale=scale, tiles=dev(tiles.reshape(-1)), n_tiles=n_tiles,
                       tile_tokens=64 if wide else 16, decode_reqs=dev(hb.decode_reqs), n_decode=len(hb.decode_reqs),
                       max_pos=max(totals), n_splits=splits, part_o=part_o, part_ml=part_ml, tensor_cores=mma, chunk=chunk or 0, **two)
    K().check_status(torch.device(DEV))
    want = torch.empty(n_tok, H, dv, dtype=torch.float64)
    maps_of = torch.empty(n_tok, H, 2, dv, dtype=torch.float64)
    t0 = 0
    for r in range(n_req):
        kc, vc = ks[r].to(dt).double(), vs[r].to(dt).double()  # what the cache holds
        qq = torch.zeros(totals[r], H, maps, dk, dtype=torch.float64)
        qq[lens_old[r]:] = q[t0:t0 + lens_new[r]].double()
        if maps == 2:
            both = P.two_maps(qq, kc, vc, scale, chunk)[lens_old[r]:]
            maps_of[t0:t0 + lens_new[r]] = both
            want[t0:t0 + lens_new[r]] = P.combine_maps(both, lam, diff, eps)
        else:
            want[t0:t0 + lens_new[r]] = one_map(qq[:, :, 0], kc[:, :, 0], vc, scale, chunk)[lens_old[r]:]
        t0 += lens_new[r]
    return out.float().cpu().view(n_tok, H, dv), want, vs, maps_of


def _tol(dtype, mma=False):
    # with bfloat16 operands on the tensor cores the queries and the probabilities are rounded too, and the difference of
    # two maps that nearly cancel (a first token's, a chunk's first) is brought to unit size
    return 3e-5 if dtype == "float32" else (5e-2 if mma else 1.5e-2)


SIZES = ((6, 2, 20, 12, 16), (5, 5, 8, 8, 8), (40, 1, 8, 8, 32), (2, 1, 136, 130, 16), (16, 4, 64, 128, 16), (3, 3, 48, 96, 16),
         (8, 8, 128, 128, 16), (7, 1, 9, 5, 8), (12, 3, 32, 64, 16), (4, 2, 16, 120, 32))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [1, 7, 16, 17, 64, 100, None])
@pytest.mark.parametrize("maps", [2, 1])
def test_attention_of_one_and_two_maps_over_chunks(dtype, chunk, maps):
    """Chunks of one key, within a page, of a page and one more, of a key tile, of several, and none; portions that start
    inside a page or chunk and cross several chunks beside single tokens; one to forty heads a key/value head; CUDA
    cores and tensor cores."""
    for mma in ((False,) if dtype == "float32" else (False, True)):
        for H, G, dk, dv, page in SIZES:
            got, want, _, _ = _attn_case(dtype, H, G, dk, dv, [40, 1, 2, 17, 1, 16], [5, 130, 0, 15, 0, 16], page, 0.3, chunk,
                                         seed=H, mma=mma, maps=maps)
            assert rel(got, want) < _tol(dtype, mma), (H, G, dk, dv, mma)
            got, want, _, _ = _attn_case(dtype, H, G, dk, dv, [1, 1, 1, 1], [0, 31, 64, 300], page, 0.2, chunk, seed=H + 50,
                                         mma=mma, maps=maps)
            assert rel(got, want) < _tol(dtype, mma), (H, G, dk, dv, mma, "single tokens")


@pytest.mark.parametrize("chunk", [None, 70, 128, 257])
@pytest.mark.parametrize("maps", [2, 1])
def test_long_portions_on_the_tensor_cores(chunk, maps):
    """Portions of one to many key tiles whose chunks begin inside a tile and at its border."""
    for H, G, dk, dv, page in ((4, 2, 64, 64, 16), (4, 1, 48, 24, 8), (4, 2, 128, 128, 16), (3, 3, 16, 120, 32), (2, 2, 64, 128, 16)):
        got, want, _, _ = _attn_case("bfloat16", H, G, dk, dv, [200, 1, 2, 65, 64, 400], [5, 130, 0, 63, 64, 330], page, 0.25, chunk,
                                     seed=H, mma=True, maps=maps)
        assert rel(got, want) < _tol("bfloat16", True), (H, G, dk, dv)


@pytest.mark.parametrize("lam,diff", [(0.0, 0.0), (1.0, 0.5), (-0.8, 0.9), (3.0, -0.5)])
def test_factors_of_the_second_map(lam, diff):
    for dtype, mma, splits in (("float32", False, 1), ("float32", False, 4), ("bfloat16", True, 1)):
        got, want, _, _ = _attn_case(dtype, 6, 3, 24, 16, [1, 20, 1, 3], [200, 9, 0, 64], 16, 0.25, 50, seed=3, splits=splits, mma=mma,
                                     lam=lam, diff=diff, eps=0.05)
        # lambda 1: where a query sees one key the maps cancel to nothing, and eps alone is under the root
        assert float((got - want).abs().max()) < (3e-5 if dtype == "float32" else 0.12), (dtype, splits)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("splits", [2, 3, 8, 32])
@pytest.mark.parametrize("chunk", [40, 512, None])
def test_decoded_tokens_with_keys_cut_into_parts(dtype, splits, chunk):
    """The maps' parts are put together before the difference, whatever their number (more parts than tiles of keys
    too), beside a prompt portion that is not cut."""
    for H, G, dk, dv in ((6, 2, 20, 10), (3, 3, 64, 128), (16, 1, 8, 200)):
        got, want, _, _ = _attn_case(dtype, H, G, dk, dv, [1, 1, 5, 1, 1], [700, 0, 40, 63, 79], 16, 0.25, chunk, seed=splits,
                                     splits=splits)
        assert rel(got, want) < _tol(dtype), (H, G)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [1, 5, 16, 33, 64, 200, None])
@pytest.mark.parametrize("which", [0, 1])
def test_a_key_that_stands_out_just_inside_the_chunk_just_outside_and_far_back(dtype, chunk, which):
    """One key is scored far above the rest in one map.  As the first key of the query's chunk (with no chunks: as the
    sequence's first key, hundreds back, and at a page's border), that map is (nearly) its value; one position earlier,
    in the chunk before, it must leave no trace.  From a prompt portion's last query (CUDA cores and tensor cores) and
    from a decoded token's (whole and cut into parts); the query at a chunk's last, first and some other place."""
    H, G, dk, dv, head = 4, 2, 24, 16, 3
    lam, diff, eps = 0.6, 0.25, 1e-3
    c = chunk or 10 ** 6
    for total in {min(c, 40) + 3, 333, 10 * c if c < 70 else 500, (400 // c) * c + 1, 897}:
        last = total - 1
        for new, splits, mma in ((min(4, total), 1, False), (min(4, total), 1, True), (1, 1, False), (1, 5, False), (min(total, 70), 1, True)):
            old = total - new
            edge = last // c * c
            cases = [(edge, True), (edge - 1, False)] if chunk else [(0, True), (last - (last % 16) - 1, True)]
            for key, inside in cases:
                if key < 0:
                    continue
                got, want, vs, maps_of = _attn_case(dtype, H, G, dk, dv, [new], [old], 16, 0.5, chunk, seed=key + 1,
                                                    stand_out=(key, head, which), splits=splits, mma=mma, lam=lam, diff=diff, eps=eps)
                rows = slice(-1, None) if mma and dtype == "bfloat16" else slice(None)
                assert rel(got[rows], want[rows]) < _tol(dtype, mma), (total, new, splits, mma, key, inside)
                value = vs[0][key, head // (H // G)].to(DTYPES[dtype]).double()
                maps = maps_of[-1, head].clone()
                near = float((maps[which] - value).abs().max())  # of the plain map itself
                if inside:
                    assert near < 1e-3
                    maps[which] = value
                    assert float((got[-1, head] - P.combine_maps(maps, lam, diff, eps)).abs().max()) < 2 * _tol(dtype, mma)
                elif last - edge >= 2:
                    maps[which] = value
                    assert float((got[-1, head] - P.combine_maps(maps, lam, diff, eps)).abs().max()) > 0.2, "a key of the chunk before was seen"


def test_refused_attention_arguments():
    lam = torch.ones(1, device=DEV)
    pool = torch.zeros(4, 1, 2, 16, 24, device=DEV)
    i = torch.zeros(4, dtype=torch.int32, device=DEV)
    t = torch.zeros(2, 4, dtype=torch.int32, device=DEV)
    base = dict(n_heads=2, dk=8, dv=8, v_at=16, scale=1.0, decode_reqs=i, n_decode=1, max_pos=16)
    q, out = torch.zeros(1, 32, device=DEV), torch.zeros(1, 16, device=DEV)
    with pytest.raises(K().KernelError):  # a sink has no place beside two maps
        K().bias_attention(q, None, pool, t, i, i, i, out, maps=2, diff_lambda=lam, sink=torch.zeros(2, device=DEV), **base)
    with pytest.raises(K().KernelError):
        K().bias_attention(q, None, pool, t, i, i, i, out, maps=3, diff_lambda=lam, **base)
    with pytest.raises(K().KernelError):  # the value lies where the second key ends
        K().bias_attention(q, None, pool, t, i, i, i, out, maps=2, diff_lambda=lam, **dict(base, v_at=8))


# ---- whole models through the step function ------------------------------------------------------------

@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("vebotar"))
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
    reqs = requests_for(name, [1, 2, 5, 16, 17, 33, 150, 300], 1)
    tr = R.whole(reqs)
    check(f, reqs, tr, replay(f, name, dtype, tr, tmp_path), dtype)


def test_every_layer_against_the_plain_streams(folders):
    """The sum of the stream's copies after each layer, in 32 bits."""
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
                kept = ctx.extras.get("stream_copies")
                caught.append((x if kept is None else kept[0].sum(1)).detach().cpu().clone())
            layer.block.forward = wrapped
        toks = requests_for(name, [45], 11)["r0"]
        slot = runner.cache.new_request()
        runner.step([StepEntry(slot, toks, [len(toks) - 1])])
        runner.check_status()
        cfg, w = load_folder(f)
        streams = []
        P.forward(cfg, w, toks, streams=streams)
        assert len(caught) == len(streams) == len(cfg["layers"])
        for i, (mine, want) in enumerate(zip(caught, streams)):
            assert rel(mine, want) < 2e-5, (name, i)


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
    for sizes in ((7, 2, 16, 3, 2, 5, 33, 2, 1, 17), (2,), (15, 1, 16, 17)):
        tr = R.portions(reqs, sizes=sizes)
        got = replay(f, name, dtype, tr, tmp_path / f"s{len(sizes)}{sizes[0]}")
        check(f, reqs, tr, got, dtype)


@pytest.mark.parametrize("graphs", [False, True], ids=["walked", "graphs"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(TINY))
def test_mixed_batches_with_pages_and_slots_used_again(folders, tmp_path, name, dtype, graphs):
    """Up to four live requests, portions beside single tokens, in a pool so small that pages and slots come
    round again; every row is compared with the request run alone (the plain implementation knows no batch): a
    key left over by a page's earlier owner, or a page a chunk gave back too early, would show."""
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
    for name in ("B", "A"):
        reqs = requests_for(name, [420], 10)
        tr = R.tail_decoded(reqs, tail=417)
        f = folders[name, dtype]
        check(f, reqs, tr, replay(f, name, dtype, tr, tmp_path / f"long{name}", cuda_graphs=True), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wide_model_with_long_contexts(tmp_path, dtype):
    """Width 1024: the products' tensor-core paths, prompts of 600 and 350 tokens whole and in portions of up to 256, the
    last tokens one by one, chunks of many key tiles."""
    folder = write_tiny("WIDE", str(tmp_path), decisive=dtype == "bfloat16")
    rng = np.random.default_rng(3)
    reqs = {f"r{i}": rng.integers(0, WIDE["raw"]["vocab"], size=n).tolist() for i, n in enumerate([600, 350])}
    for i, tr in enumerate((R.whole(reqs), R.tail_decoded(reqs, tail=6), R.portions(reqs, sizes=(256, 3, 130, 64, 200)))):
        wanted = {rid: {len(t) - 1, len(t) - 2, len(t) // 2, 299, 300, 0, 1} for rid, t in reqs.items()}
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
    decode graphs): every generated token is the plain arg-max given the tokens before it, or within the precision's
    reach."""
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


def test_preemption_changes_no_token(folders):
    """A pool too small for four requests at once: the one admitted last gives its pages back and is recomputed; the
    tokens are those of a run with room for all."""
    from rosellm_b200.engine.llm import InferenceEngine

    f = folders["F", "float32"]  # no chunks: a request holds all its pages
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

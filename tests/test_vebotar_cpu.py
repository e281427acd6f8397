"""Vebotar without a GPU: configuration, refusals, the spec it builds, tensor names, what the cache keeps for layers
that read other layers' keys under other masks, and the plain implementation's mechanisms on cases small enough to
work out by hand."""
import copy
import math
import random

import pytest
import torch

import plain_vebotar as P
from tiny_vebotar import TINY, WIDE, attn, load_folder, model, write_tiny

from rosellm_b200.cache import CacheManager
from rosellm_b200.config.base import ConfigError, parse_config, resolve_architecture
from rosellm_b200.config.vebotar import VebotarConfig
from rosellm_b200.models.model import Model, named_params_of_spec
from rosellm_b200.parts import KVCacheSpec
from rosellm_b200.parts.standard import scaled_rotary_frequencies
from rosellm_b200.weights.loader import WeightError, match_tensors


def spec_of(raw):
    cfg = parse_config(raw)
    return cfg, resolve_architecture(cfg.to_dict()).build_spec(cfg)


@pytest.mark.parametrize("name", list(TINY) + ["WIDE"])
def test_configuration_round_trip_and_spec(name):
    raw = WIDE["raw"] if name == "WIDE" else TINY[name]["raw"]
    cfg, spec = spec_of(raw)
    assert isinstance(cfg, VebotarConfig) and VebotarConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == raw
    assert [r.layer for r in spec.run_order] == list(range(len(raw["layers"])))
    assert [r.cache_of for r in spec.run_order] == [l["mixer"].get("kv_from") for l in raw["layers"]]
    assert spec.head.kind == "linear" and spec.embedding.params["scale"] == raw["embedding"]["scale"]
    for lr, ls in zip(raw["layers"], spec.layers):
        names = [n for n, _, _ in ls.parts]
        assert (lr["mlp"] is None) == ("feed_forward" not in names) == ("connect_feed_forward" not in names)
        assert ls.block.kind == "hyper_connections" and ls.block.params["copies"] == raw["streams"]
        mixer, mx = ls.part("mixer"), lr["mixer"]
        assert mixer.kind == "differential_attention" and mixer.params["chunk"] == (mx.get("mask") or {}).get("size")
        assert mixer.params["own_kv"] == ("kv_from" not in mx) == ("k_weight" in mixer.tensors)
        assert mixer.params["diff"] == mx["diff"] and mixer.params["rot_dims"] == (mx.get("rot") or {"dims": 0})["dims"]
        if lr["mlp"] is not None:
            ff = ls.part("feed_forward")
            assert ff.params["score"] == "chosen_softmax" and ff.params["gate"] == "relu_squared"
            assert ff.params["shared_inner"] == (lr["mlp"].get("shared") or {"ff": 0})["ff"]


def test_refusals():
    raw = TINY["A"]["raw"]
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "kv_heads"), 4), (("width",), 60),
                        (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "dims"), 18),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("norm", "eps"), 0.0), (("streams",), 0),
                        (("layers", 0, "mlp", "router", "top"), 6), (("layers", 0, "mlp", "kind"), "dense"),
                        (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0), (("layers", 0, "mlp", "shared", "ff"), 0),
                        (("layers", 0, "mixer", "rot", "base"), 1.0), (("layers", 1, "mixer", "kv_from"), 1),
                        (("layers", 1, "mixer", "kv_from"), -1), (("layers", 3, "mixer", "kv_from"), 1),
                        (("layers", 3, "mixer", "kv_from"), 0), (("layers", 1, "mixer", "dim"), 12)):
        bad = copy.deepcopy(raw)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises((ConfigError, ValueError)):
            cfg, spec = spec_of(bad)
            Model(spec, torch.float32, "cpu")
    with pytest.raises(ValueError):
        _, spec = spec_of(dict(TINY["E"]["raw"], streams=17))
        Model(spec, torch.float32, "cpu")


def test_tensor_names(tmp_path):
    folder = write_tiny("A", str(tmp_path))
    raw, tensors = load_folder(folder)
    assert {"embed", "final.norm", "head", "l0.norm1", "l0.norm2", "l0.hc1.in", "l0.hc1.out", "l0.hc1.mix", "l0.hc2.mix",
            "l0.mix.q", "l0.mix.k", "l0.mix.v", "l0.mix.lq1", "l0.mix.lk2", "l0.mix.o", "l0.mlp.router", "l0.mlp.e4.down",
            "l0.mlp.shared.sg", "l1.mix.q", "l2.norm1"} <= set(tensors)
    assert not {"l1.mix.k", "l1.mix.v", "l3.mix.k", "l2.norm2", "l2.hc2.in", "l3.mlp.shared.sg"} & set(tensors)
    assert tensors["l0.mix.q"].shape == (6 * 2 * 16, 64) and tensors["l0.mix.k"].shape == (2 * 2 * 16, 64)
    assert tensors["l0.mix.v"].shape == (2 * 24, 64) and tensors["l0.mix.o"].shape == (64, 6 * 24)
    assert tensors["l0.hc1.mix"].shape == (3, 3) and tensors["l0.mlp.shared.sg"].shape == (1, 64)
    _, spec = spec_of(raw)
    tensors = {k: v.float() for k, v in tensors.items()}
    match_tensors(named_params_of_spec(spec), tensors, source="test")
    for missing in ("l1.mix.lq2", "l0.mlp.e3.up", "l0.mlp.shared.sg", "l2.hc1.out"):
        with pytest.raises(WeightError):
            match_tensors(named_params_of_spec(spec), {k: v for k, v in tensors.items() if k != missing}, source="test")
    with pytest.raises(WeightError):  # a tensor that no part reads
        match_tensors(named_params_of_spec(spec), dict(tensors, **{"l1.mix.k": tensors["l0.mix.k"]}), source="test")


def test_factor_of_the_second_map():
    m = Model(spec_of(TINY["A"]["raw"])[1], torch.float32, "cpu")
    g = torch.Generator().manual_seed(1)
    part = m.layers[1].mixer
    t = {r: torch.randn(16, generator=g) * 0.4 for r in ("lq1", "lk1", "lq2", "lk2")}
    part.bind({"q_weight": torch.zeros(6 * 2 * 16, 64), "out_weight": torch.zeros(64, 6 * 24), **t})
    want = P.difference_factor(*(t[r].double() for r in ("lq1", "lk1", "lq2", "lk2")), 0.6)
    assert float(part.diff_lambda) == pytest.approx(float(want), rel=1e-6) and abs(float(want) - 0.6) > 0.05


# ---- what the cache keeps -----------------------------------------------------------------------------------

def test_specs_of_shared_caches_cover_every_reader():
    """A cache that several layers read is kept for the one that sees farthest back: layer 0 of A alone would keep its
    chunk of 7, layer 1 reads the same pages in chunks of 50; in B the reader sees all keys."""
    kv = Model(spec_of(TINY["A"]["raw"])[1], torch.float32, "cpu").kv_specs()
    assert set(kv) == {0, 2}
    assert kv[0] == KVCacheSpec(2, 2 * 16 + 24, None, planes=1, chunks=(7, 50))
    assert kv[2] == KVCacheSpec(4, 2 * 24 + 8, None, planes=1, chunks=(5, 16))
    kv = Model(spec_of(TINY["B"]["raw"])[1], torch.float32, "cpu").kv_specs()
    assert set(kv) == {0, 2} and not kv[0].bounded and kv[2].chunks == (100,)
    assert kv[0].head_dim == 32  # two keys of 9 entries, the value of 5 from entry 24 on
    kv = Model(spec_of(TINY["D"]["raw"])[1], torch.float32, "cpu").kv_specs()
    assert kv[0].chunks == (48, 96) and kv[1].chunks == (128,) and set(kv) == {0, 1}
    raw = model(50, 16, 1e-5, 1.0, 2, [(attn(2, 2, 8, 8, 0.3, 0.5, 4), None), (attn(4, 2, 8, 8, 0.3, 0.5, 4, kv_from=0), None)])
    Model(spec_of(raw)[1], torch.float32, "cpu").kv_specs()  # more query heads than the source: the rows are the same


def test_first_key_in_sight():
    for spec, sees in ((KVCacheSpec(1, 8, None), lambda i, j: True), (KVCacheSpec(1, 8, 5), lambda i, j: i - j < 5),
                       (KVCacheSpec(1, 8, None, chunks=(7,)), lambda i, j: i // 7 == j // 7),
                       (KVCacheSpec(1, 8, None, chunks=(4, 6)), lambda i, j: i // 4 == j // 4 or i // 6 == j // 6),
                       (KVCacheSpec(1, 8, 3, chunks=(10,)), lambda i, j: i - j < 3 or i // 10 == j // 10)):
        for pos in range(60):
            # the earliest key that any query from pos on sees, by looking at them all
            want = min(j for i in range(pos, pos + 30) for j in range(i + 1) if sees(i, j))
            assert spec.first_key(pos) == want, (spec, pos)
            if spec.bounded:
                assert pos - spec.first_key(pos) < spec.reach
    a, b = KVCacheSpec(1, 8, None, chunks=(7,)), KVCacheSpec(1, 8, 5)
    assert a.covering(b) == KVCacheSpec(1, 8, 5, chunks=(7,)) and a.covering(KVCacheSpec(1, 8, None)).bounded is False
    assert a.covering(a) == a and not a.same_rows(KVCacheSpec(2, 8, None)) and a.same_rows(b)


def test_pages_of_passed_chunks_come_back_while_the_request_lives():
    """Random portions and decoded tokens of several requests on one pool: every key a later query sees keeps its page,
    a page that no query sees is given back, none is lost or held twice."""
    rng = random.Random(3)
    for page, chunks in ((4, (6,)), (8, (8,)), (16, (5,)), (4, (6, 20)), (8, (1,)), (4, (16,))):
        spec = KVCacheSpec(2, 16, None, planes=1, chunks=chunks)
        m = CacheManager({0: spec, 1: spec}, {}, page_size=page, num_pages=64, max_slots=3, max_seq_len=200, device="cpu")
        live = {}
        for _ in range(400):
            if len(live) < 3 and rng.random() < 0.3:
                live[m.new_request()] = 0
            if not live:
                continue
            slot = rng.choice(list(live))
            n = min(rng.choice([1, 1, 1, 2, 3, 7, 20]), 200 - live[slot])
            if n == 0 or rng.random() < 0.02:
                m.release(slot)
                del live[slot]
                continue
            assert m.reserve(slot, n)
            row = m.groups[0].table[slot]
            for i in range(live[slot], live[slot] + n):  # every page a token of this step reads or writes is there
                assert all(row[j // page] >= 0 for j in range(spec.first_key(i), i + 1) if j >= 0)
            m.commit(slot, n)
            live[slot] += n
            assert all(p < 0 for p in m.groups[0].table[slot][:spec.first_key(live[slot]) // page])
            assert len(m.pages_of(slot)) <= -(-spec.reach // page) + 1
            m.check()
        for slot in list(live):
            m.release(slot)
        m.check()
        assert m.num_free_pages == 64


def test_scheduler_plans_pages_of_chunked_layers():
    from rosellm_b200.engine.scheduler import Scheduler

    spec = KVCacheSpec(1, 8, None, planes=1, chunks=(8,))
    m = CacheManager({0: spec}, {}, page_size=4, num_pages=8, max_slots=2, max_seq_len=400, device="cpu")
    s = Scheduler(m, max_num_seqs=2, max_num_batched_tokens=8, prefill_chunk_size=8, max_model_len=400)
    assert s._pages_to_hold(300) == [-(-(8 + 8) // 4) + 1]  # far fewer than 300 tokens take


# ---- the plain implementation by hand -------------------------------------------------------------------------

def test_plain_ramp_against_the_package_and_by_hand():
    for dims, base in ((8, 500.0), (24, 9000.0), (2, 1.0e6), (64, 20000.0)):
        f, mult = P.ramp_frequencies(dims, base, None)
        assert mult == 1.0 and f == pytest.approx([base ** (-2 * i / dims) for i in range(dims // 2)])
        for factor, original, fast, slow in ((4.0, 24, 6.0, 1.0), (16.0, 512, 32.0, 1.0), (3.0, 24, 6.0, 5.9), (8.0, 20, 4.0, 0.5)):
            sc = dict(factor=factor, original=original, fast=fast, slow=slow)
            want, want_mult = P.ramp_frequencies(dims, base, sc)
            got, got_mult = scaled_rotary_frequencies(dims, base, dict(sc, kind="ramp"))
            assert got.tolist() == pytest.approx(want, rel=1e-6) and got_mult == pytest.approx(want_mult)
            assert want_mult == pytest.approx(1 + 0.1 * math.log(factor))
    # dims 8, base 10^4: pair i turns original / (2 pi 10^i) times; the ramp runs from pair 0 to pair 2
    f, _ = P.ramp_frequencies(8, 1.0e4, dict(factor=4.0, original=64, fast=4.0, slow=0.25))
    assert f == pytest.approx([1.0, 0.1 * (0.5 / 4 + 0.5), 0.01 / 4, 0.001 / 4])


def test_plain_turn_mask_and_maps_by_hand():
    y = torch.tensor([[[1.0, 0.0, 2.0, 0.0, 5.0, 6.0]]], dtype=torch.float64).repeat(3, 1, 1)
    out = P.turn(y, torch.arange(3), [1.0, 0.1], 2.0)
    for p in range(3):
        assert out[p, 0].tolist() == pytest.approx([2 * math.cos(p), 2 * math.sin(p), 4 * math.cos(p * 0.1), 4 * math.sin(p * 0.1), 5.0, 6.0])
    assert P.seen_keys(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    assert torch.equal(P.seen_keys(5, None), P.seen_keys(5, 5)) and torch.equal(P.seen_keys(4, 1), torch.eye(4).bool())
    # equal scores: both maps average the values in sight
    T = 6
    q, k = torch.zeros(T, 2, 2, 3, dtype=torch.float64), torch.zeros(T, 1, 2, 3, dtype=torch.float64)
    v = torch.arange(T, dtype=torch.float64).view(T, 1, 1)
    o = P.two_maps(q, k, v, 1.0, 3)
    assert o[:, 1, 1, 0].tolist() == pytest.approx([0.0, 0.5, 1.0, 3.0, 3.5, 4.0])
    # one score stands out in the second map alone
    q[5, 0, 1, 0], k[3, 0, 1, 0] = 40.0, 1.0
    o = P.two_maps(q, k, v, 1.0, 3)
    assert o[5, 0, :, 0].tolist() == pytest.approx([4.0, 3.0])
    maps = torch.tensor([[[3.0, 0.0], [1.0, 2.0]]], dtype=torch.float64)
    d = torch.tensor([3.0 - 0.5, -1.0], dtype=torch.float64)
    want = d / math.sqrt(float((d * d).mean()) + 0.25) * 0.2
    assert P.combine_maps(maps, 0.5, 0.8, 0.25)[0].tolist() == pytest.approx(want.tolist())
    one = torch.tensor([math.log(2.0), 0.0], dtype=torch.float64)
    other = torch.tensor([0.0, math.log(3.0)], dtype=torch.float64)
    unit_row = torch.ones(2, dtype=torch.float64)
    assert float(P.difference_factor(one, unit_row, other, unit_row, 0.25)) == pytest.approx(2.0 - 3.0 + 0.25)


def test_plain_experts_and_streams_by_hand():
    z = torch.tensor([[0.0, math.log(3.0), -5.0, math.log(1.0) + 0.0]], dtype=torch.float64)
    idx, weight = P.route(torch.tensor([[0.0, math.log(3.0), -5.0]], dtype=torch.float64), 2)
    assert idx.tolist() == [[1, 0]] and weight[0].tolist() == pytest.approx([0.75, 0.25])
    assert P.route(z, 1)[1].tolist() == [[1.0]]
    h = torch.tensor([[2.0, -1.0]], dtype=torch.float64)
    eye = torch.eye(2, dtype=torch.float64)
    assert P.squared_relu_mlp(h, eye * 3.0, eye)[0].tolist() == [36.0, 0.0]
    w = {"m.router": torch.tensor([[0.0, 0.0], [math.log(3.0) / 2, 0.0], [0.0, 9.0]], dtype=torch.float64)}
    for e in range(3):
        w[f"m.e{e}.up"], w[f"m.e{e}.down"] = eye, eye * 10.0 ** e
    out = P.experts(h, w, "m.", {"router": {"experts": 3, "top": 2}})
    assert out[0].tolist() == pytest.approx([0.25 * 4.0 + 0.75 * 40.0, 0.0])
    w.update({"m.shared.up": -eye, "m.shared.down": eye, "m.shared.sg": torch.tensor([[0.0, -math.log(3.0)]], dtype=torch.float64)})
    out = P.experts(h, w, "m.", {"router": {"experts": 3, "top": 2}, "shared": {"ff": 2}})
    assert out[0].tolist() == pytest.approx([31.0, 0.75])  # the shared expert sees (-2, 1): 1, times sigmoid(ln 3)
    X = torch.tensor([[[1.0]], [[10.0]]], dtype=torch.float64)
    M = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=torch.float64)
    assert P.read_streams(X, torch.tensor([2.0, 0.5], dtype=torch.float64)).item() == 7.0
    new = P.write_streams(X, M, torch.tensor([100.0, 200.0], dtype=torch.float64), torch.tensor([[1.0]], dtype=torch.float64))
    assert new.flatten().tolist() == [1 + 30 + 100, 2 + 40 + 200]


def test_plain_layers_that_share_keys(tmp_path):
    """The second layer of E reads the first's keys and values: giving it projections of its own that equal the first's
    would be another model, since its input differs."""
    cfg, w = load_folder(write_tiny("E", str(tmp_path)))
    toks = [3, 50, 7, 7, 12, 80]
    shared = P.forward(cfg, w, toks)
    own = copy.deepcopy(cfg)
    del own["layers"][1]["mixer"]["kv_from"]
    w2 = dict(w, **{"l1.mix.k": w["l0.mix.k"], "l1.mix.v": w["l0.mix.v"]})
    assert float((P.forward(own, w2, toks) - shared).abs().max()) > 0.1

"""Kugadra without a GPU: configuration, refusals, the spec it builds, tensor names, what the cache and the state slots
hold, the reordering that serves rotations in halves, and the plain implementation's mechanisms on cases small enough to
work out by hand."""
import copy
import math

import pytest
import torch

import plain_kugadra as P
from tiny_kugadra import TINY, WIDE, latent, load_folder, model, write_tiny

from rosellm_b200.config.base import ConfigError, parse_config, resolve_architecture
from rosellm_b200.config.kugadra import KugadraConfig
from rosellm_b200.models.model import Model, named_params_of_spec
from rosellm_b200.parts import KVCacheSpec
from rosellm_b200.parts.base import build_part
from rosellm_b200.parts.standard import RotaryPositions
from rosellm_b200.weights.loader import WeightError, match_tensors


def spec_of(raw):
    cfg = parse_config(raw)
    return cfg, resolve_architecture(cfg.to_dict()).build_spec(cfg)


@pytest.mark.parametrize("name", list(TINY) + ["WIDE"])
def test_configuration_round_trip_and_spec(name):
    raw = WIDE["raw"] if name == "WIDE" else TINY[name]["raw"]
    cfg, spec = spec_of(raw)
    assert isinstance(cfg, KugadraConfig) and KugadraConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == raw
    assert [r.layer for r in spec.run_order] == list(range(len(raw["layers"])))
    assert [r.cache_of for r in spec.run_order] == [l["mixer"].get("kv_from") for l in raw["layers"]]
    assert spec.head.kind == "tied_to_embedding" and spec.head.params["soft_cap"] == raw["logit_softcap"]
    assert spec.embedding.params["scale"] == raw["embedding"]["scale"]
    for lr, ls in zip(raw["layers"], spec.layers):
        names = [n for n, _, _ in ls.parts]
        assert ls.block.kind == "pre_post_norm" and (lr["mlp"] is None) == ("feed_forward" not in names)
        mixer, mx = ls.part("mixer"), lr["mixer"]
        if lr["type"] == "lightning":
            assert mixer.kind == "lightning_attention" and list(mixer.params["decay"]) == mx["decay"]
        else:
            assert mixer.kind == "latent_attention" and mixer.params["gate"] == "head" and mixer.params["rot_pairs"] == "halves"
            assert mixer.params["own_kv"] == ("kv_from" not in mx) == ("dkv_weight" in mixer.tensors)
            assert mixer.params["scale"] == mx["scale"] and mixer.params["sink"] is False
        if lr["mlp"] is not None and lr["mlp"]["kind"] == "moe":
            ff = ls.part("feed_forward")
            assert ff.params["weight_scale"] == lr["mlp"]["router"]["scale"] and ff.params["correction"]
            assert ff.params["shared_inner"] == (lr["mlp"].get("shared") or {"ff": 0})["ff"]
        elif lr["mlp"] is not None:
            ff = ls.part("feed_forward")
            assert ff.kind == "dense_mlp" and ff.params["activation"] == "relu_squared" and not ff.params["bias"]


def test_refusals():
    raw = TINY["A"]["raw"]
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "decay"), [0.5, 0.5]), (("width",), 60),
                        (("layers", 0, "mixer", "decay"), [0.5, 1.5, 0.1]), (("layers", 0, "mixer", "dim"), 300),
                        (("layers", 1, "mixer", "rot_dim"), 5), (("layers", 1, "mixer", "rot", "dims"), 4), (("norm", "eps"), 0.0),
                        (("logit_softcap",), 0.0), (("layers", 1, "mlp", "router", "top"), 6), (("layers", 1, "mlp", "kind"), "glu"),
                        (("layers", 1, "mlp", "router", "scale"), 0.0), (("layers", 1, "mlp", "shared", "ff"), 0),
                        (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0), (("layers", 1, "mixer", "rot", "base"), 1.0),
                        (("layers", 2, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_from"), 0),
                        (("layers", 1, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_rank"), 12),
                        (("layers", 2, "mixer", "rot", "base"), 500.0), (("layers", 1, "mixer", "kv_rank"), 600)):
        bad = copy.deepcopy(raw)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises((ConfigError, ValueError)):
            cfg, spec = spec_of(bad)
            Model(spec, torch.float32, "cpu")
    missing = copy.deepcopy(raw)
    del missing["layers"][1]["mixer"]["q_rank"]
    with pytest.raises(ConfigError):
        spec_of(missing)
    common = dict(hidden_size=16, num_heads=2, plain_dim=8, rot_dim=4, value_dim=8, kv_rank=8, scale=1.0, rot_dims=4,
                  rot_base=100.0, norm_eps=1e-5)
    from rosellm_b200.parts.latent import LatentAttention

    for bad in (dict(gate="row"), dict(rot_pairs="thirds")):
        with pytest.raises(ValueError):
            LatentAttention(**common, **bad)


def test_tensor_names(tmp_path):
    folder = write_tiny("A", str(tmp_path))
    raw, tensors = load_folder(folder)
    assert {"embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.q", "l0.mix.k", "l0.mix.v",
            "l0.mix.g", "l0.mix.norm", "l0.mix.o", "l0.mlp.up", "l0.mlp.down", "l1.mix.dq", "l1.mix.dq.norm", "l1.mix.uq",
            "l1.mix.dkv", "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.uv", "l1.mix.g", "l1.mix.o", "l1.mlp.router",
            "l1.mlp.correction", "l1.mlp.e4.gate", "l1.mlp.e0.up", "l1.mlp.e2.down", "l1.mlp.shared.gate", "l1.mlp.shared.up",
            "l1.mlp.shared.down", "l2.mix.uk", "l2.norm1b"} <= set(tensors)
    assert not {"head", "l2.mix.dkv", "l2.mix.dkv.norm", "l2.norm2", "l3.mlp.shared.up", "l0.mlp.gate"} & set(tensors)
    assert tensors["l0.mix.g"].shape == (3 * 20, 64) and tensors["l0.mix.norm"].shape == (3 * 20,)
    assert tensors["l1.mix.uq"].shape == (4 * 18, 20) and tensors["l1.mix.dkv"].shape == (18 + 6, 64)
    assert tensors["l1.mix.g"].shape == (4, 64) and tensors["l2.mix.uv"].shape == (7 * 14, 18)
    _, spec = spec_of(raw)
    tensors = {k: v.float() for k, v in tensors.items()}
    match_tensors(named_params_of_spec(spec), tensors, source="test", ignored=spec.ignored_tensors)
    match_tensors(named_params_of_spec(spec), dict(tensors, **{"l2.norm2": torch.ones(64)}), source="test", ignored=spec.ignored_tensors)
    for missing in ("l0.mix.norm", "l1.mlp.e3.up", "l1.mlp.correction", "l2.mix.dq.norm", "l1.mix.dkv"):
        with pytest.raises(WeightError):
            match_tensors(named_params_of_spec(spec), {k: v for k, v in tensors.items() if k != missing}, source="test",
                          ignored=spec.ignored_tensors)
    with pytest.raises(WeightError):  # a tensor that no part reads
        match_tensors(named_params_of_spec(spec), dict(tensors, **{"l2.mix.dkv": tensors["l1.mix.dkv"]}), source="test",
                      ignored=spec.ignored_tensors)


def test_what_the_cache_and_the_state_slots_hold():
    """A layer that reads another's rows has none of its own; linear attention keeps a float32 state and no pages."""
    m = Model(spec_of(TINY["A"]["raw"])[1], torch.bfloat16, "cpu")
    assert m.kv_specs() == {1: KVCacheSpec(1, 24, None, planes=1)}
    states = m.state_specs()
    assert {k: (s.shape, s.dtype) for k, s in states.items()} == {0: ((3, 12, 20), torch.float32), 3: ((2, 24, 8), torch.float32)}
    m = Model(spec_of(TINY["B"]["raw"])[1], torch.float32, "cpu")
    assert set(m.kv_specs()) == {0} and set(m.state_specs()) == {2}
    with pytest.raises(ValueError):  # rows of another form
        spec = spec_of(model(50, 16, 1e-5, 1.0, 5.0, [(latent(2, 8, 4, 8, 12, 8, 0.3, (10.0,)), None),
                                                      (latent(2, 8, 4, 8, 12, 8, 0.3, (10.0,), kv_from=0), None)]))[1]
        import dataclasses

        layer = spec.layers[1]
        parts = tuple((n, c, dataclasses.replace(s, params=dict(s.params, kv_rank=20)) if n == "mixer" else s) for n, c, s in layer.parts)
        Model(dataclasses.replace(spec, layers=(spec.layers[0], dataclasses.replace(layer, parts=parts))), torch.float32, "cpu").kv_specs()


def test_powers_of_the_decays():
    part = build_part("mixer", spec_of(TINY["A"]["raw"])[1].layers[3].part("mixer"))
    pw = part.decay_powers()
    assert pw.shape == (2, 65) and pw[0].eq(1.0).all()
    assert float(pw[1, 0]) == 1.0 and pw[1, 1:].eq(0.0).all()
    part = build_part("mixer", spec_of(TINY["A"]["raw"])[1].layers[0].part("mixer"))
    assert part.decay_powers()[1].tolist() == pytest.approx([0.93 ** n for n in range(65)], rel=1e-6)


@pytest.mark.parametrize("name,layer", [("A", 1), ("B", 0), ("D", 1), ("E", 0)])
def test_rotation_in_halves_by_reordered_rows(name, layer):
    """The part turns neighbouring pairs of reordered rows: queries and key parts projected by the bound weights and
    turned in pairs hold the same numbers, reordered alike, as the file's weights turned in halves."""
    spec = spec_of(TINY[name]["raw"])[1]
    part = build_part("mixer", spec.layers[layer].part("mixer"))
    g = torch.Generator().manual_seed(layer)
    t = {p.role: torch.randn(p.shape, generator=g, dtype=torch.float64) for p in part.param_specs()}
    part.bind(dict(t))
    T, H, dn, dr = 6, part.num_heads, part.plain_dim, part.rot_dim
    pos = torch.tensor([0, 1, 5, 40, 333, 1000])
    cq, h = torch.randn(T, part.q_rank, generator=g, dtype=torch.float64), torch.randn(T, part.hidden_size, generator=g, dtype=torch.float64)
    q_file, q_bound = (cq @ t["q_weight"].T).view(T, H, dn + dr), (cq @ part.q_weight[:, :part.q_rank].T).view(T, H, dn + dr)
    at = part.offsets["dkv"]
    k_file, k_bound = h @ t["dkv_weight"].T, h @ part.proj_weight[at:at + part.kv_rank + dr].T
    assert torch.equal(q_file[..., :dn], q_bound[..., :dn]) and torch.equal(k_file[:, :part.kv_rank], k_bound[:, :part.kv_rank])
    if dr == 0:
        return
    m = TINY[name]["raw"]["layers"][layer]["mixer"]
    freqs, mult = P.rotation_constants(m["rot"])
    rotary = RotaryPositions(dims=dr, base=m["rot"]["base"], scaling=part.rotary.scaling)
    assert rotary.frequencies("cpu").tolist() == pytest.approx(freqs, rel=1e-6) and rotary.mult == pytest.approx(mult)

    def pairs(y):
        out = y.clone()
        for i, f in enumerate(freqs):
            c, s = (fn(pos.double() * f) * mult for fn in (torch.cos, torch.sin))
            shape = [T] + [1] * (y.dim() - 2)
            a, b = y[..., 2 * i], y[..., 2 * i + 1]
            out[..., 2 * i], out[..., 2 * i + 1] = a * c.view(shape) - b * s.view(shape), b * c.view(shape) + a * s.view(shape)
        return out

    want_q, want_k = P.rotate_halves(q_file[..., dn:], pos, freqs, mult), P.rotate_halves(k_file[:, part.kv_rank:], pos, freqs, mult)
    got_q, got_k = pairs(q_bound[..., dn:]), pairs(k_bound[:, part.kv_rank:])
    n = dr // 2
    order = [i for p in range(n) for i in (p, p + n)]
    assert torch.allclose(got_q, want_q[..., order], atol=1e-12) and torch.allclose(got_k, want_k[:, order], atol=1e-12)


# ---- the plain implementation by hand ---------------------------------------------------------------------------

def test_plain_states_by_hand():
    one = lambda *x: torch.tensor(x, dtype=torch.float64).view(-1, 1, 1)
    o, S = P.decayed_states(one(1, 1, 2), one(3, 5, 7), one(1, 10, 100), [0.5])
    assert o.flatten().tolist() == [3.0, 1.5 + 50.0, 2 * (0.75 + 25.0 + 700.0)] and S.item() == 725.75
    o2, S2 = P.decayed_states(one(1), one(0), one(0), [0.5], state=S)
    assert o2.item() == S2.item() == 725.75 / 2
    q = torch.tensor([[[1.0, 2.0]]], dtype=torch.float64)
    o, S = P.decayed_states(q, torch.tensor([[[3.0, 4.0]]], dtype=torch.float64), torch.tensor([[[5.0, 6.0, 7.0]]], dtype=torch.float64), [0.9])
    assert o[0, 0].tolist() == [55.0, 66.0, 77.0] and S[0].tolist() == [[15.0, 18.0, 21.0], [20.0, 24.0, 28.0]]
    assert P.silu(torch.tensor(0.0)).item() == 0.0 and P.silu(torch.tensor(2.0)).item() == pytest.approx(2 / (1 + math.exp(-2)))


def test_plain_rotation_and_ramp_by_hand():
    y = torch.tensor([[1.0, 2.0, 0.0, 0.0, 9.0]], dtype=torch.float64).repeat(3, 1)
    out = P.rotate_halves(y, torch.arange(3), [1.0, 0.1], 2.0)
    for p in range(3):
        assert out[p].tolist() == pytest.approx([2 * math.cos(p), 4 * math.cos(0.1 * p), 2 * math.sin(p), 4 * math.sin(0.1 * p), 9.0])
    # dims 8, base 10^4, original 2 pi 10^3: a pair that turns t times has index 3 - log10 t; fast 100 -> 1, slow 1 -> 3
    f, mult = P.rotation_constants({"dims": 8, "base": 10000.0, "scaling": {"factor": 4.0, "original": 2000.0 * math.pi, "fast": 99.0, "slow": 1.01}})
    assert mult == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert f == pytest.approx([1.0, 0.1, 0.01 * (0.5 / 4 + 0.5), 0.001 / 4])
    assert P.rotation_constants({"dims": 4, "base": 100.0}) == ([1.0, 0.1], 1.0)


def test_plain_choice_feed_forwards_and_bound_by_hand():
    z = torch.log(torch.tensor([0.5, 0.3, 0.2], dtype=torch.float64))
    none = torch.zeros(3, dtype=torch.float64)
    ids, a = P.choose(z, none, 2, 1.0)
    assert ids == [0, 1] and a.tolist() == pytest.approx([0.625, 0.375])
    ids, a = P.choose(z, torch.tensor([-0.4, 0.0, 0.05], dtype=torch.float64), 2, 3.0)  # choice scores 0.1, 0.3, 0.25
    assert ids == [1, 2] and a.tolist() == pytest.approx([1.8, 1.2])
    eye = torch.eye(2, dtype=torch.float64)
    h = torch.tensor([[2.0, -1.0]], dtype=torch.float64)
    assert P.dense(h, {"m.up": eye * 3.0, "m.down": eye}, "m.")[0].tolist() == [36.0, 0.0]
    s = 2 / (1 + math.exp(-2))
    w = {"m.router": torch.tensor([[0.0, 0.0], [math.log(3.0) / 2, 0.0]], dtype=torch.float64), "m.correction": none[:2]}
    for e in range(2):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"] = eye, eye, eye * 10.0 ** e
    mlp = {"router": {"experts": 2, "top": 1, "scale": 0.5}}
    assert P.experts(h, w, "m.", mlp)[0, 0].item() == pytest.approx(0.5 * 10 * s * 2)
    w.update({"m.shared.gate": eye, "m.shared.up": -eye, "m.shared.down": eye})
    assert P.experts(h, w, "m.", dict(mlp, shared={"ff": 2}))[0, 0].item() == pytest.approx(0.5 * 10 * s * 2 - 2 * s)
    assert P.soft_cap(torch.tensor([0.0, 3.0, 1e9], dtype=torch.float64), 3.0).tolist() == pytest.approx([0.0, 3 * math.tanh(1.0), 3.0])


def test_plain_layers_that_share_latents(tmp_path):
    """The second layer of E reads the first's latents: giving it a W_dkv that equals the first's would be another model,
    since its input differs."""
    cfg, w = load_folder(write_tiny("E", str(tmp_path)))
    toks = [3, 50, 7, 7, 12, 80]
    shared = P.forward(cfg, w, toks)
    own = copy.deepcopy(cfg)
    del own["layers"][1]["mixer"]["kv_from"]
    w2 = dict(w, **{"l1.mix.dkv": w["l0.mix.dkv"], "l1.mix.dkv.norm": w["l0.mix.dkv.norm"]})
    assert float((P.forward(own, w2, toks) - shared).abs().max()) > 0.05

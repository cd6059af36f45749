"""Kulesun without a GPU: the configuration and its spec, tensor names, the caches a model asks for, the plain
implementation's own consistency."""
import copy
import math

import pytest
import torch

import plain_kulesun as plain
from kulesun_cases import CASES, draw_case


def _cfg(d):
    from gogguf_b200.config import config_from_dict
    return config_from_dict(copy.deepcopy(d))


def _weights(d, seed=1, std=0.12):
    from gogguf_b200.engine.model import expected_tensors
    from gogguf_b200.weights.loader import random_tensors
    return random_tensors(expected_tensors(_cfg(d).to_spec()), seed, std, 0.1, dtype=torch.float32)


@pytest.mark.parametrize("name", sorted(CASES))
def test_config_round_trip_and_spec(name):
    from gogguf_b200.engine.model import expected_tensors
    d = CASES[name][0]
    cfg = _cfg(d)
    assert cfg.to_dict() == d
    spec = cfg.to_spec()
    assert len(spec.schedule) == len(spec.blocks) == len(d["layers"])
    decl = {n: t for n, t in expected_tensors(spec).items() if not t.optional}
    assert {"embed", "final.norm"} <= set(decl) and "head" not in decl          # the head is the embedding table
    sources = 0
    for i, l in enumerate(d["layers"]):
        p = f"l{i}."
        own = ({"q", "dkv", "dkv.norm", "uk", "uv", "g", "o"} if l["type"] == "latent_attention" else
               {"q", "q.b", "k", "k.b", "v", "v.b", "talk", "g", "o", "o.b"} | ({"vmix"} if l["mixer"]["v_mix"] else set()))
        assert {n[len(p) + 4:] for n in decl if n.startswith(p + "mix.")} == own
        for n in ("norm2", "norm2b", "mlp.gate", "mlp.up", "mlp.down"):
            assert (p + n in decl) == (l["mlp"] is not None)
        assert {p + "norm1", p + "norm1b"} <= set(decl)
        if l["mixer"].get("v_mix"):
            mix = spec.blocks[i].parts["mixer"]["value_mix"]
            assert mix == ("mix" if sources else "source")
            sources += 1
    assert cfg.parameter_count() == sum(math.prod(t.shape) for t in decl.values())


def test_shapes_follow_the_configuration():
    from gogguf_b200.engine.model import expected_tensors
    t = expected_tensors(_cfg(CASES["S"][0]).to_spec())
    assert t["l0.mix.q"].shape == (3 * 26, 80) and t["l0.mix.dkv"].shape == (34, 80) and t["l0.mix.uk"].shape == (60, 28)
    assert t["l0.mix.uv"].shape == (36, 28) and t["l0.mix.g"].shape == (36, 80) and t["l0.mix.dkv.norm"].shape == (28,)
    assert t["l1.mix.q"].shape == (72, 80) and t["l1.mix.k"].shape == (24, 80) and t["l1.mix.v"].shape == (40, 80)
    assert t["l1.mix.q.b"].shape == (72,) and t["l1.mix.o.b"].shape == (80,) and t["l1.mix.talk"].shape == (6, 6)
    assert t["l1.mix.g"].shape == (6, 80) and t["l1.mix.vmix"].shape == () and "l3.mix.vmix" not in t


@pytest.mark.parametrize("bad", [
    lambda d: d["layers"][0].update(type="other"),
    lambda d: d["layers"][1]["mixer"].update(kv_heads=4),                      # 6 heads over 4 kv heads
    lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8),                   # beyond the rotated part
    lambda d: d["layers"][0]["mixer"]["rot"].update(dims=3),
    lambda d: d["layers"][0]["mixer"]["rot"].update(base=1.0),
    lambda d: d["layers"][0]["mixer"].pop("rot"),
    lambda d: d["layers"][0]["mixer"].pop("scale"),
    lambda d: d["layers"][4]["mixer"].update(vdim=24),                         # another size than the source of values
    lambda d: d["layers"][4]["mixer"].update(kv_heads=4),
    lambda d: d["layers"][1]["mixer"].update(softcap=-1.0),
    lambda d: d["layers"][1]["mixer"].update(v_mix=1),
    lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=0),
    lambda d: d["layers"][1]["mixer"]["q_temp"].pop("coef"),
    lambda d: d["layers"][0]["mlp"].update(kind="moe"),
    lambda d: d["layers"][0]["mlp"].update(ff=0),
    lambda d: d["norm"].update(eps=0.0),
    lambda d: d.update(layers=[]),
    lambda d: d.pop("width"),
])
def test_a_bad_configuration_is_refused(bad):
    from gogguf_b200.config import ConfigError
    d = copy.deepcopy(CASES["S"][0])
    bad(d)
    with pytest.raises(ConfigError):
        _cfg(d)


def test_what_the_layers_cache():
    from gogguf_b200.cache.sequence_cache import KVRequest, LatentRequest
    from gogguf_b200.parts.latent_attention import LatentAttentionMixer
    from gogguf_b200.parts.mixed_head_attention import MixedHeadAttentionMixer
    spec = _cfg(CASES["S"][0]).to_spec()
    assert LatentAttentionMixer.cache_request(spec.blocks[0].parts["mixer"]) == LatentRequest(width=34, window=None)
    assert (MixedHeadAttentionMixer.cache_request(spec.blocks[1].parts["mixer"])
            == KVRequest(num_kv_heads=2, head_dim=12, window=None, value_dim=20))
    assert _cfg(CASES["S"][0]).kv_bytes_per_token(4) == 4 * (34 + 2 * 32 + 30 + 3 * 24 + 2 * 48 + 2 * 28)


# ----------------------------------------------------------------------------------------------- the oracle itself
def test_softmax_with_one_in_its_denominator():
    s = torch.tensor([[2.0, -math.inf], [-50.0, -60.0], [300.0, 299.0]], dtype=torch.float64)
    p = plain.weights_with_one(s)
    assert abs(float(p[0, 0]) - math.exp(2) / (1 + math.exp(2))) < 1e-15 and float(p[0, 1]) == 0.0
    assert float(p[1].sum()) < 1e-20                                  # nothing is worth looking at: all weights vanish
    assert abs(float(p[2].sum()) - 1.0) < 1e-12 and bool(torch.isfinite(p).all())


def test_temperature_steps_where_it_should():
    t = plain.query_temperature(10, 0.5, 4)
    assert [round(float(v), 6) for v in t[:3]] == [1.0, 1.0, 1.0]
    assert abs(float(t[3]) - (1 + 0.5 * math.log(2))) < 1e-15 and float(t[6]) == float(t[3])
    assert abs(float(t[7]) - (1 + 0.5 * math.log(3))) < 1e-15


def test_mixing_the_weights_is_mixing_the_results_on_every_kv_head():
    g = torch.Generator().manual_seed(2)
    H, G, n, dv = 6, 2, 5, 4
    a = torch.rand(H, n, n, generator=g, dtype=torch.float64)
    T = torch.randn(H, H, generator=g, dtype=torch.float64)
    v = torch.randn(n, G, dv, generator=g, dtype=torch.float64)
    own = [h // (H // G) for h in range(H)]
    want = torch.einsum("hij,jhe->ihe", plain.talking(a, T), v[:, own])
    u = torch.einsum("gij,jce->igce", a, v)
    got = torch.stack([torch.einsum("g,ige->ie", T[h], u[:, :, own[h]]) for h in range(H)], dim=1)
    assert float((got - want).abs().max()) < 1e-12


def test_rotation_in_halves_keeps_lengths_and_depends_on_the_distance():
    rot = dict(dims=8, base=100.0, scaling=dict(factor=4.0, original=64, fast=16.0, slow=2.0))
    _, mag = plain.yarn_frequencies(rot)
    g = torch.Generator().manual_seed(3)
    q, k = (torch.randn(1, 10, generator=g, dtype=torch.float64).repeat(9, 1) for _ in range(2))
    qr, kr = plain.rotate_halves(q, rot), plain.rotate_halves(k, rot)
    assert float((qr[:, :8].norm(dim=1) - mag * q[:, :8].norm(dim=1)).abs().max()) < 1e-12
    assert torch.equal(qr[:, 8:], q[:, 8:])
    assert abs(float(qr[5] @ kr[2] - qr[8] @ kr[5])) < 1e-12 and abs(float(qr[5] @ kr[2] - qr[5] @ kr[3])) > 1e-3


@pytest.mark.parametrize("name", ["S", "ONE"])
def test_a_prefix_does_not_see_what_comes_after(name):
    d = CASES[name][0]
    w = _weights(d)
    tokens = [int(t) for t in torch.randint(0, d["vocab"], (40,), generator=torch.Generator().manual_seed(5))]
    whole = plain.forward(d, w, tokens)
    for n in (1, 2, 17):
        assert float((plain.forward(d, w, tokens[:n]) - whole[:n]).abs().max()) < 1e-10


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations_are_valid(seed):
    d = draw_case(seed)
    cfg = _cfg(d)
    assert cfg.to_dict() == d
    out = plain.forward(d, _weights(d), [1, 2, 3])
    assert out.shape == (3, d["vocab"]) and bool(torch.isfinite(out).all())


def test_random_weights_of_the_new_kinds():
    w = _weights(CASES["S"][0])
    t = w["l1.mix.talk"]
    assert t.shape == (6, 6) and float((t - torch.eye(6)).abs().mean()) > 0.05 and float(t.diagonal().mean()) > 0.5
    assert 0.1 < float(w["l1.mix.vmix"]) < 0.9 and w["l1.mix.vmix"].shape == ()

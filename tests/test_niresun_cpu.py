"""Niresun without a GPU: the configuration and its spec, tensor names, the caches a model asks for, the plain
implementation's own consistency."""
import copy
import math

import pytest
import torch

import plain_niresun as plain
from niresun_cases import CASES, draw_case


def _cfg(d):
    from gogguf_b200.config import config_from_dict
    return config_from_dict(copy.deepcopy(d))


def _weights(d, seed=1, std=0.12):
    from gogguf_b200.engine.model import expected_tensors
    from gogguf_b200.weights.loader import random_tensors
    return random_tensors(expected_tensors(_cfg(d).to_spec()), seed, std, 0.1, dtype=torch.float32)


OWN = {"mamba1": {"in", "conv", "conv.b", "x", "dt", "dt.b", "A_log", "D", "o"},
       "attention": {"q", "q.b", "k", "k.b", "v", "v.b", "g", "o"},
       "parallel": {"left." + n for n in ("q", "k", "v", "q.conv", "k.conv", "v.conv", "o", "out")}
       | {"right." + n for n in ("q", "k", "v", "g", "i", "i.b", "f", "f.b", "norm", "o", "out")}}


@pytest.mark.parametrize("name", sorted(CASES))
def test_config_round_trip_and_spec(name):
    from gogguf_b200.engine.model import expected_tensors
    d = CASES[name][0]
    cfg = _cfg(d)
    assert cfg.to_dict() == d
    spec = cfg.to_spec()
    assert len(spec.schedule) == len(spec.blocks) == len(d["layers"])
    decl = {n: t for n, t in expected_tensors(spec).items() if not t.optional}
    assert {"embed", "head", "final.norm", "final.norm.alpha", "final.norm.b"} <= set(decl)
    for i, l in enumerate(d["layers"]):
        p = f"l{i}."
        assert {n[len(p) + 4:] for n in decl if n.startswith(p + "mix.")} == OWN[l["type"]]
        for n in ("norm2", "norm2.alpha", "norm2.b", "mlp.gate", "mlp.up", "mlp.down"):
            assert (p + n in decl) == (l["mlp"] is not None)
        assert {p + "norm1", p + "norm1.alpha", p + "norm1.b"} <= set(decl)
    assert cfg.parameter_count() == sum(math.prod(t.shape) for t in decl.values())


def test_shapes_follow_the_configuration():
    from gogguf_b200.engine.model import expected_tensors
    t = expected_tensors(_cfg(CASES["S"][0]).to_spec())
    shapes = {
        "l0.mix.left.q": (72, 76), "l0.mix.left.k": (24, 76), "l0.mix.left.v": (40, 76), "l0.mix.left.v.conv": (40, 4),
        "l0.mix.left.o": (76, 120), "l0.mix.left.out": (76,), "l0.mix.right.q": (30, 76), "l0.mix.right.g": (42, 76),
        "l0.mix.right.i": (3, 76), "l0.mix.right.f.b": (3,), "l0.mix.right.norm": (42,), "l0.mix.right.o": (76, 42),
        "l1.mix.in": (104, 76), "l1.mix.conv": (52, 4), "l1.mix.x": (13, 52), "l1.mix.dt": (52, 3), "l1.mix.A_log": (52, 5),
        "l1.mix.D": (52,), "l1.mix.o": (76, 52), "l2.mix.q.b": (72,), "l2.mix.g": (40, 76), "l2.mix.v": (20, 76),
        "l0.norm1.alpha": (), "head": (197, 76)}
    assert {n: t[n].shape for n in shapes} == shapes


@pytest.mark.parametrize("bad", [
    lambda d: d["layers"][0].update(type="other"),
    lambda d: d["layers"][0]["mixer"].pop("right"),
    lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4),              # 6 heads over 4 kv heads
    lambda d: d["layers"][0]["mixer"]["left"]["q_temp"].update(every=0),
    lambda d: d["layers"][0]["mixer"]["left"]["q_temp"].pop("coef"),
    lambda d: d["layers"][0]["mixer"]["right"].update(gate_cap=0.0),
    lambda d: d["layers"][1]["mixer"].update(state=0),
    lambda d: d["layers"][1]["mixer"].pop("dt_rank"),
    lambda d: d["layers"][1]["mixer"].update(conv=True),
    lambda d: d["layers"][2]["mixer"].pop("mask"),
    lambda d: d["layers"][2]["mixer"]["mask"].update(size=0),
    lambda d: d["layers"][2]["mixer"]["rot"].update(dims=20),                  # beyond the head
    lambda d: d["layers"][2]["mixer"]["rot"].update(dims=3),
    lambda d: d["layers"][2]["mixer"]["rot"]["scaling"].pop("low"),
    lambda d: d["layers"][2]["mixer"].pop("scale"),
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
    from gogguf_b200.cache.sequence_cache import KVRequest, KVView, SequenceCache, StateView
    from gogguf_b200.parts.registry import MIXERS
    spec = _cfg(CASES["S"][0]).to_spec()
    req = [MIXERS[b.parts["mixer"].kind].cache_request(b.parts["mixer"]) for b in spec.blocks]
    (tail, kv), (S, n, m) = req[0]
    assert kv == KVRequest(num_kv_heads=2, head_dim=12, value_dim=20) and tail.shape == (3, 136)
    assert (S.shape, n.shape, m.shape) == ((3, 10, 14), (3, 10), (3,))
    assert [r.shape for r in req[1]] == [(3, 52), (52, 5)]
    assert req[2] == KVRequest(num_kv_heads=2, head_dim=18, value_dim=10, chunk=37)
    one = _cfg(CASES["ONE"][0]).to_spec()
    req1 = [MIXERS[b.parts["mixer"].kind].cache_request(b.parts["mixer"]) for b in one.blocks]
    assert req1[0][0] is None and isinstance(req1[1][0], KVRequest)             # one tap keeps nothing
    cache = SequenceCache(req, [None] * len(req), max_tokens=256, dtype=torch.float32)
    left, right = cache.view(0)
    assert isinstance(left[0], StateView) and isinstance(left[1], KVView) and len(right) == 3
    assert left[1].k.shape[-1] == 12 and left[1].v.shape[-1] == 20 and right[0].state.shape[1:] == (3, 10, 14)
    # a state is zeroed when its slot is opened again; nothing can be cut back
    s = cache.open()
    right[2].state[s] = 5.0
    cache.plan([s], [3]); cache.commit([s], [3])
    assert not cache.truncate(s, 2)
    cache.close(s)
    while cache.open() != s:
        pass
    assert float(right[2].state[s].abs().max()) == 0.0


def test_a_chunked_layer_gives_its_pages_back_as_chunks_end():
    from gogguf_b200.cache.sequence_cache import KVRequest, SequenceCache
    cache = SequenceCache([KVRequest(1, 8, chunk=100), KVRequest(1, 8)], [None, None], max_tokens=64 * 8, dtype=torch.float32)
    g = cache.groups[0]
    s = cache.open()
    held = {}
    for n in range(1, 321):
        cache.plan([s], [1]); cache.commit([s], [1])
        held[n] = [i for i, p in enumerate(g.seq_pages[s]) if p >= 0]
        first = n // 100 * 100                         # what the token at position n reads
        assert all(i in held[n] for i in range(first // 64, (n + 63) // 64)), n
        cache.check()
    assert held[99] == [0, 1] and held[100] == [1] and held[199] == [1, 2, 3] and held[200] == [3] and held[320] == [4]
    assert not cache.truncate(s, 250) and cache.truncate(s, 310)       # position 250's chunk starts in a page given back
    cache.close(s)
    assert g.pages.held_count == 0
    w = SequenceCache([KVRequest(1, 8, window=70)], [None], max_tokens=64 * 8, dtype=torch.float32)
    s = w.open()
    w.plan([s], [200]); w.commit([s], [200])
    assert [i for i, p in enumerate(w.groups[0].seq_pages[s]) if p >= 0] == [2, 3]


# ----------------------------------------------------------------------------------------------- the oracle itself
def test_frequencies_keep_slow_down_and_mix():
    rot = dict(dims=64, base=10000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=512))
    f, g = plain.frequencies(dict(dims=64, base=10000.0)), plain.frequencies(rot)
    turns = 512 * f / (2 * math.pi)
    assert torch.equal(g[turns > 4], f[turns > 4]) and bool((g[turns < 1] == f[turns < 1] / 8).all())
    mid = (turns >= 1) & (turns <= 4)
    assert int(mid.sum()) > 2 and bool(((g < f) & (g > f / 8))[mid].all())
    from gogguf_b200.parts.base import Runtime
    from gogguf_b200.parts.position import RotaryBanded
    p = RotaryBanded(dict(theta=10000.0, rotary_dim=64, factor=8.0, low=1.0, high=4.0, original=512),
                     Runtime(dtype=torch.float32, device=torch.device("cpu")))
    assert float((p.inv_freq - g).abs().max()) < 1e-15


def test_chunks_count_from_the_start():
    m = plain.unseen(8, torch.float64, 3)
    see = [[j for j in range(8) if m[i, j] == 0] for i in range(8)]
    assert see == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6], [6, 7]]


def test_convolution_meets_the_token_with_its_last_tap():
    u = torch.tensor([[1.0], [10.0], [100.0]])
    assert plain.causal_conv(u, torch.tensor([[2.0, 3.0]])).flatten().tolist() == [3.0, 32.0, 320.0]
    assert plain.causal_conv(u[:1], torch.tensor([[1.0, 2.0, 3.0, 4.0]]), torch.tensor([0.5])).flatten().tolist() == [4.5]


def test_memory_is_the_sum_it_stands_for():
    """Without the maximum: o = sum_j e^(F_i - F_j + i_j) (q . k_j) v_j over the larger of the like sum's size and one."""
    g = torch.Generator().manual_seed(2)
    n, H, d, dv = 9, 2, 3, 4
    q, k = (torch.randn(n, H, d, generator=g, dtype=torch.float64) for _ in range(2))
    v = torch.randn(n, H, dv, generator=g, dtype=torch.float64)
    i = torch.randn(n, H, generator=g, dtype=torch.float64) * 3
    f = -torch.rand(n, H, generator=g, dtype=torch.float64)
    F = f.cumsum(0)
    got = plain.memory_scan(q, k, v, i, f)
    for t in range(n):
        wt = torch.exp(F[t] - F[:t + 1] + i[:t + 1]) * torch.einsum("jhd,hd->jh", k[:t + 1], q[t])
        m = torch.maximum(F[t], (F[t] - F[:t + 1] + i[:t + 1]).max(0).values)
        den = torch.maximum(wt.sum(0).abs(), torch.ones(H, dtype=torch.float64)) + 1e-6 * torch.exp(m)
        want = torch.einsum("jh,jhe->he", wt, v[:t + 1]) / den[:, None]
        assert float((got[t] - want).abs().max()) < 1e-12


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


def test_rows_per_chunk_of_a_selective_scan():
    from gogguf_b200.parts.linear_recurrent import selective_chunk
    assert selective_chunk(2048, 1, 4096, 16) == 128 and selective_chunk(2048, 8, 4096, 16) == 0      # enough to fill the GPU
    assert selective_chunk(200, 1, 256, 16) == 64 and selective_chunk(2048, 64, 256, 24) == 0
    assert selective_chunk(1, 1, 256, 16) == 0 and selective_chunk(100, 1, 256, 16) == 0

"""Tiny Kulesun configurations for the tests, model folders made from them, and the plain implementation's view of a
folder.  The configurations differ from one another in every size, in the order of their layers and in their
constants; some take values that another model may happen to make equal or one."""
from __future__ import annotations

import os
from typing import Dict, List, Optional

import torch


def rot(dims, base, scaling=None):
    d = dict(dims=dims, base=base)
    if scaling is not None:
        d["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return d


def attn(heads, kv_heads, dim, vdim, scale, softcap=None, q_temp=None, v_mix=True):
    d = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if softcap:
        d["softcap"] = softcap
    if q_temp:
        d["q_temp"] = dict(coef=q_temp[0], every=q_temp[1])
    return d


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, rotation):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=rotation)


def layer(mixer, ff):
    return dict(type="latent_attention" if "kv_rank" in mixer else "attention", mixer=mixer,
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def model(vocab, width, eps, layers, emb=1.0, logit=1.0):
    return dict(architecture="Kulesun", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb),
                logit_scale=logit, layers=layers)


# sizes no tensor-core kernel takes; a source of values that is not the first layer; layers of three kinds of sharing
# (source, mixing, neither), without bound, without temperature, without feed-forward; rotations with and without
# stretched frequencies
CASE_S = model(211, 80, 2e-6, [
    layer(latent(3, 20, 6, 12, 28, 0.25, rot(6, 10000.0, (4.0, 64, 16.0, 2.0))), 56),
    layer(attn(6, 2, 12, 20, 0.3, 15.0, (0.5, 7.0)), None),
    layer(latent(5, 12, 10, 36, 20, 0.4, rot(10, 700.0)), 24),
    layer(attn(3, 3, 16, 8, 0.5, v_mix=False), 40),
    layer(attn(4, 2, 28, 20, 0.2, 3.0, (0.2, 3.0)), 100),
    layer(attn(2, 2, 8, 20, 0.6, None, (-0.1, 11.0)), None),
], emb=3.5, logit=0.7)
# values that happen to be one or equal: one head, one kv head, equal key and value sizes, factors of one, a
# temperature that changes with every token, a rotated part of two
CASE_ONE = model(97, 64, 1e-5, [
    layer(attn(1, 1, 16, 16, 1.0, 30.0, (1.0, 1.0)), 48),
    layer(latent(1, 16, 2, 16, 16, 0.3, rot(2, 50.0, (1.0, 32, 8.0, 1.0))), None),
    layer(attn(1, 1, 16, 16, 0.25, 1.0), 16),
])
# sizes the tensor-core kernels take: wide matrices, rows on 16-byte boundaries; heads that do not fill a tile evenly
CASE_W = model(523, 384, 3e-6, [
    layer(attn(6, 2, 64, 96, 0.125, 20.0, (0.3, 50.0)), 512),
    layer(latent(4, 64, 32, 64, 128, 0.1, rot(32, 40000.0, (3.0, 256, 16.0, 1.0))), 256),
    layer(attn(10, 2, 40, 96, 0.2, 8.0, (0.1, 9.0)), 128),
    layer(latent(6, 48, 16, 112, 64, 0.15, rot(16, 1e6)), None),
    layer(attn(3, 3, 128, 128, 0.08, None, None, v_mix=False), 192),
], emb=12.5, logit=1.5)

CASES = {"S": (CASE_S, 3), "ONE": (CASE_ONE, 4), "W": (CASE_W, 6)}
# the wide case's matrices are drawn smaller, so that its products neither grow nor shrink what they are given: with
# larger ones its scores are so large that the rounding of bfloat16 alone moves whole rows
STD = {"S": 0.12, "ONE": 0.12, "W": 0.05}


def write_case(tmp, tag: str, cfg: dict, seed: int, store_dtype: str = "float32", std: float = 0.12,
               norm_std: float = 0.1) -> str:
    from gogguf_b200.config import config_from_dict
    from gogguf_b200.engine.model import write_random_model
    folder = os.path.join(str(tmp), f"kulesun_{tag}_{store_dtype}_{std}")
    if not os.path.isdir(folder):
        write_random_model(config_from_dict(cfg), seed, folder, dtype=store_dtype, std=std, norm_std=norm_std)
    return folder


def make_folder(tmp, name: str, store_dtype: str = "float32", std: Optional[float] = None, norm_std: float = 0.1) -> str:
    """Write case `name` with the product's random-weights mode; returns the folder."""
    cfg, seed = CASES[name]
    return write_case(tmp, name, cfg, seed, store_dtype, STD[name] if std is None else std, norm_std)


def plain_logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
                 dtype=torch.float64):
    import plain_kulesun as plain
    return plain.forward(cfg, w, tokens, dtype, layers_out)


def rounded_logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """The plain implementation in float64 with the inputs and outputs of its projections rounded to bfloat16: how far
    rounding alone moves each row of this model."""
    import plain_kulesun as plain
    exact = plain.linear
    r = lambda x: x.to(torch.bfloat16).to(x.dtype)
    plain.linear = lambda x, w_, name, bias=False: r(exact(r(x), w_, name, bias))
    try:
        return plain.forward(cfg, w, tokens, torch.float64)
    finally:
        plain.linear = exact


def draw_case(seed: int) -> dict:
    """A configuration nobody chose: every size, the order of the layers and the constants from a seeded generator."""
    import random
    r = random.Random(seed)
    width = r.choice([24, 40, 64, 120, 200])
    G, vdim = r.choice([1, 2, 3]), r.choice([4, 8, 24, 40, 64, 128])      # what the layers that share values agree on
    layers = []
    for _ in range(r.choice([1, 2, 3, 4, 5])):
        ff = None if r.random() < 0.25 else r.choice([8, 40, 128, 200])
        if r.random() < 0.5:
            rd = r.choice([2, 4, 16, 32])
            sc = None if r.random() < 0.4 else (r.choice([1.5, 2.0, 8.0]), r.choice([32, 100, 512]), r.choice([8.0, 32.0]),
                                                r.choice([0.5, 1.0, 2.0]))
            m = latent(r.choice([1, 2, 5, 8]), r.choice([4, 16, 32, 40]), rd, r.choice([4, 16, 48, 80]),
                       r.choice([8, 16, 36, 64, 160]), r.choice([0.1, 0.3]), rot(rd, r.choice([100.0, 10000.0, 1e6]), sc))
        else:
            share = r.random() < 0.8
            g = G if share else r.choice([1, 2, 4])
            dim = r.choice([4, 8, 20, 32, 64, 128])
            m = attn(g * r.choice([1, 2, 4, 5]), g, dim, vdim if share else r.choice([8, 20, 64]),
                     round(r.choice([0.3, 1.0, 2.0]) * dim ** -0.5, 4), r.choice([None, 5.0, 30.0]),
                     r.choice([None, (0.5, 4.0), (0.1, 100.0), (2.0, 1.0)]), v_mix=share)
        layers.append(layer(m, ff))
    return model(r.choice([53, 211, 641]), width, r.choice([1e-6, 1e-5, 3e-4]), layers, r.choice([1.0, 7.0]),
                 r.choice([1.0, 0.3, 4.0]))

"""Tiny Niresun configurations for the tests, model folders made from them, and the plain implementation's view of a
folder.  The configurations differ from one another in every size, in the order of their layers and in their
constants; some take values that another model may happen to make equal or one."""
from __future__ import annotations

import os
from typing import Dict, List, Optional

import torch


def rot(dims, base, scaling=None):
    d = dict(dims=dims, base=base)
    if scaling is not None:
        d["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return d


def chunked(heads, kv_heads, dim, vdim, scale, size, rotation):
    d = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size))
    if rotation is not None:
        d["rot"] = rotation
    return d


def left(heads, kv_heads, dim, vdim, scale, conv, q_temp):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, conv=conv,
                q_temp=dict(coef=q_temp[0], every=q_temp[1]))


def right(heads, dim, vdim, cap):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def mamba(inner, state, dt_rank, conv):
    return dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv)


def layer(mixer, ff):
    kind = "mamba1" if "inner" in mixer else ("parallel" if "left" in mixer else "attention")
    return dict(type=kind, mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


def pair(l, r):
    return dict(left=l, right=r)


def model(vocab, width, eps, layers):
    return dict(architecture="Niresun", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


# sizes no tensor-core kernel takes; every kind of layer with and without a feed-forward
CASE_S = model(197, 76, 2e-6, [
    layer(pair(left(6, 2, 12, 20, 0.3, 4, (0.5, 7.0)), right(3, 10, 14, 6.0)), 56),
    layer(mamba(52, 5, 3, 4), None),
    layer(chunked(4, 2, 18, 10, 0.25, 37, rot(6, 10000.0, (4.0, 1.0, 4.0, 64))), 40),
    layer(mamba(70, 11, 9, 2), 24),
    layer(pair(left(3, 3, 20, 12, 0.4, 2, (0.2, 3.0)), right(5, 18, 22, 15.0)), None),
    layer(chunked(5, 1, 14, 26, 0.3, 50, rot(14, 700.0)), None),
])
# values that happen to be one or equal: one head, one kv head, one tap, a state of one number, chunks of a page, equal key
# and value sizes, a temperature that changes with every token, a rotation of one pair
CASE_ONE = model(89, 64, 1e-5, [
    layer(mamba(32, 1, 1, 1), 48),
    layer(pair(left(1, 1, 16, 16, 1.0, 1, (1.0, 1.0)), right(1, 16, 16, 1.0)), 16),
    layer(chunked(1, 1, 16, 16, 0.25, 64, rot(2, 50.0, (1.0, 1.0, 1.0, 32))), None),
])
# sizes the tensor-core kernels take: wide matrices, rows on 16-byte boundaries, head sizes that do not fill a tile evenly
CASE_W = model(503, 384, 3e-6, [
    layer(mamba(512, 16, 24, 4), 512),
    layer(pair(left(8, 2, 64, 64, 0.125, 4, (0.3, 50.0)), right(4, 64, 128, 12.0)), 256),
    layer(chunked(6, 2, 72, 48, 0.12, 100, rot(40, 40000.0, (3.0, 1.0, 4.0, 256))), 128),
    layer(mamba(256, 40, 16, 3), None),
    layer(chunked(4, 1, 128, 128, 0.09, 70, rot(128, 1e6)), 192),
    layer(pair(left(10, 5, 40, 96, 0.15, 3, (0.1, 9.0)), right(6, 24, 40, 20.0)), None),
])

CASES = {"S": (CASE_S, 3), "ONE": (CASE_ONE, 4), "W": (CASE_W, 6)}
# the wide case's matrices are drawn smaller, so that its products neither grow nor shrink what they are given
STD = {"S": 0.12, "ONE": 0.12, "W": 0.05}


def write_case(tmp, tag: str, cfg: dict, seed: int, store_dtype: str = "float32", std: float = 0.12,
               norm_std: float = 0.1) -> str:
    from gogguf_b200.config import config_from_dict
    from gogguf_b200.engine.model import write_random_model
    folder = os.path.join(str(tmp), f"niresun_{tag}_{store_dtype}_{std}")
    if not os.path.isdir(folder):
        write_random_model(config_from_dict(cfg), seed, folder, dtype=store_dtype, std=std, norm_std=norm_std)
    return folder


def make_folder(tmp, name: str, store_dtype: str = "float32", std: Optional[float] = None, norm_std: float = 0.1) -> str:
    """Write case `name` with the product's random-weights mode; returns the folder."""
    cfg, seed = CASES[name]
    return write_case(tmp, name, cfg, seed, store_dtype, STD[name] if std is None else std, norm_std)


def plain_logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
                 dtype=torch.float64):
    import plain_niresun as plain
    return plain.forward(cfg, w, tokens, dtype, layers_out)


def rounded_logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """The plain implementation in float64 with the inputs and outputs of its projections rounded to bfloat16: how far
    rounding alone moves each row of this model.  (The recurrence's gates and the logits are left unrounded.)"""
    import plain_niresun as plain
    exact = plain.linear
    r = lambda x: x.to(torch.bfloat16).to(x.dtype)
    whole = ("right.i", "right.f", "mix.dt", "head")

    def rounded(x, w_, name, bias=False):
        y = exact(r(x), w_, name, bias)
        return y if name.endswith(whole) else r(y)
    plain.linear = rounded
    try:
        return plain.forward(cfg, w, tokens, torch.float64)
    finally:
        plain.linear = exact


def draw_case(seed: int) -> dict:
    """A configuration nobody chose: every size, the order of the layers and the constants from a seeded generator."""
    import random
    r = random.Random(seed)
    layers = []
    for _ in range(r.choice([1, 2, 3, 4, 5])):
        ff = None if r.random() < 0.3 else r.choice([8, 40, 128, 200])
        kind = r.choice(["mamba1", "parallel", "attention"])
        if kind == "mamba1":
            m = mamba(r.choice([8, 36, 64, 200, 320]), r.choice([1, 3, 8, 16, 20, 48]), r.choice([1, 4, 7, 16, 24]), r.choice([1, 2, 3, 4]))
        else:
            g, dim = r.choice([1, 2, 3]), r.choice([4, 8, 20, 32, 64, 80, 128])
            heads, vdim = g * r.choice([1, 2, 4, 5]), r.choice([4, 8, 24, 48, 64, 128])
            scale = round(r.choice([0.3, 1.0, 2.0]) * dim ** -0.5, 4)
            if kind == "attention":
                sc = None if r.random() < 0.4 else (r.choice([1.5, 2.0, 8.0]), r.choice([0.5, 1.0]), r.choice([2.0, 4.0]), r.choice([32, 100, 512]))
                m = chunked(heads, g, dim, vdim, scale, r.choice([3, 16, 40, 64, 100, 1000]),
                            rot(r.choice([x for x in (2, 4, 16, 64) if x <= dim]), r.choice([100.0, 10000.0, 1e6]), sc))
            else:
                m = pair(left(heads, g, dim, vdim, scale, r.choice([1, 2, 3, 4]), r.choice([(0.5, 4.0), (0.1, 100.0), (1.0, 1.0)])),
                         right(r.choice([1, 2, 3, 6]), r.choice([4, 8, 18, 32, 64]), r.choice([8, 20, 32, 64, 96]), r.choice([2.0, 8.0, 20.0])))
        layers.append(layer(m, ff))
    return model(r.choice([53, 211, 641]), r.choice([24, 40, 64, 120, 200]), r.choice([1e-6, 1e-5, 3e-4]), layers)

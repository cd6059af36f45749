"""A plain, slow restatement of the Kulesun decoder, one function per mechanism, on the CPU.

It shares no code with the package: tensors come in as a dict of torch tensors by name, the configuration as the
parsed config.json.  Everything is computed in the dtype asked for (float64 in the tests), one whole sequence at a
time.

Notation: x [n, W] is the residual stream of one sequence, positions 0..n-1.

    x_0 = s_e E[token]
    layer:      x <- x + N(mixer(N(x; w1)); w1b);   x <- x + N(ff(N(x; w2)); w2b)       (ff may be absent)
    N(y; w):    y / sqrt(mean(y^2) + eps) * (1 + w)
    mixer:      attention (no rotation; a temperature on q that grows with the position, values of unit root mean
                square mixed with the first such layer's, bounded scores, one in the softmax's denominator, the heads'
                weights mixed by a matrix, one gate per head) or latent attention (a gate per output element)
    ff:         W_down (silu(W_gate x) * W_up x)
    output:     logits = s_l E N(x; w_final)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch


# ----------------------------------------------------------------------------------------------- small pieces
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_about_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * (1.0 + w.to(x.dtype))


def linear(x: torch.Tensor, w: Dict[str, torch.Tensor], name: str, bias: bool = False) -> torch.Tensor:
    y = x @ w[name].to(x.dtype).t()
    return y + w[name + ".b"].to(x.dtype) if bias else y


# ----------------------------------------------------------------------------------------------- rotation
def yarn_frequencies(rot: dict) -> Tuple[torch.Tensor, float]:
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_halves(v: torch.Tensor, rot: dict) -> torch.Tensor:
    """v [n, ..., d]: the pairs (i, i + dims / 2) of the first rot.dims elements turn by position * f_i."""
    dims = int(rot["dims"])
    f, mag = yarn_frequencies(rot)
    n, half = v.shape[0], dims // 2
    ang = torch.arange(n, dtype=torch.float64)[:, None] * f[None, :]
    shape = (n,) + (1,) * (v.dim() - 2) + (half,)
    c, s = (torch.cos(ang) * mag).to(v.dtype).reshape(shape), (torch.sin(ang) * mag).to(v.dtype).reshape(shape)
    out = v.clone()
    a, b = v[..., :half], v[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


# ----------------------------------------------------------------------------------------------- attention
def query_temperature(n: int, coef: float, every) -> torch.Tensor:
    p = torch.arange(n, dtype=torch.float64)
    return 1.0 + coef * torch.log(torch.floor((p + 1.0) / every) + 1.0)


def bounded(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def weights_with_one(s: torch.Tensor) -> torch.Tensor:
    """s [..., keys] (-inf: not seen): exp(s_j) / (1 + sum_j exp(s_j))."""
    m = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def talking(weights: torch.Tensor, t: torch.Tensor) -> torch.Tensor:
    """weights [H, n, n]: head h's weights become sum_g t[h, g] weights_g."""
    return torch.einsum("hg,gij->hij", t.to(weights.dtype), weights)


def mixed_values(v: torch.Tensor, first: Optional[torch.Tensor], lam: float) -> torch.Tensor:
    return v if first is None else (1.0 - lam) * v + lam * first


def causal_scores(q: torch.Tensor, k: torch.Tensor, scale: float) -> torch.Tensor:
    """q [n, H, d], k [n, H, d] -> [H, n, n] with -inf above the diagonal."""
    n = q.shape[0]
    return torch.einsum("ihd,jhd->hij", q, k) * scale + unseen(n, q.dtype)


def unseen(n: int, dtype: torch.dtype) -> torch.Tensor:
    return torch.full((n, n), -math.inf, dtype=dtype).triu(1)


def attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float, first_values: Dict[str, torch.Tensor],
              ) -> torch.Tensor:
    """`first_values`: the step's place for the first mixing layer's values."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w, p + "q", True).reshape(n, H, d)
    k = linear(h, w, p + "k", True).reshape(n, G, d)
    v = rms_unit(linear(h, w, p + "v", True).reshape(n, G, dv), eps)
    qt = m.get("q_temp")
    if qt:
        q = q * query_temperature(n, qt["coef"], qt["every"]).to(q.dtype)[:, None, None]
    if m.get("v_mix"):
        if "v" in first_values:
            v = mixed_values(v, first_values["v"], float(w[p + "vmix"].double()))
        else:
            first_values["v"] = v
    own = [g // (H // G) for g in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, own]) * m["scale"]
    s = bounded(s, m.get("softcap") or 0.0) + unseen(n, h.dtype)
    a = talking(weights_with_one(s), w[p + "talk"])
    o = torch.einsum("hij,jhe->ihe", a, v[:, own])
    o = o * sigmoid(linear(h, w, p + "g"))[:, :, None]
    return linear(o.reshape(n, H * dv), w, p + "o", True)


def latent_attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(h, w, p + "q").reshape(n, H, d + r)
    dkv = linear(h, w, p + "dkv")
    c = rms_unit(dkv[:, :R], eps) * w[p + "dkv.norm"].to(h.dtype)
    k_rot = rotate_halves(dkv[:, R:], m["rot"])
    q_rot = rotate_halves(q[..., d:], m["rot"])
    k = linear(c, w, p + "uk").reshape(n, H, d)
    v = linear(c, w, p + "uv").reshape(n, H, dv)
    s = torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    a = torch.softmax(s * m["scale"] + unseen(n, h.dtype), dim=-1)
    o = torch.einsum("hij,jhe->ihe", a, v).reshape(n, H * dv)
    return linear(o * sigmoid(linear(h, w, p + "g")), w, p + "o")


# ----------------------------------------------------------------------------------------------- the rest
def feed_forward(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return linear(silu(linear(h, w, p + "gate")) * linear(h, w, p + "up"), w, p + "down")


def layer(i: int, l: dict, w: Dict[str, torch.Tensor], x: torch.Tensor, eps: float, first_values: dict) -> torch.Tensor:
    p = f"l{i}."
    h = norm_about_one(x, w[p + "norm1"], eps)
    if l["type"] == "attention":
        y = attention(l["mixer"], w, p + "mix.", h, eps, first_values)
    else:
        y = latent_attention(l["mixer"], w, p + "mix.", h, eps)
    x = x + norm_about_one(y, w[p + "norm1b"], eps)
    if l["mlp"] is not None:
        x = x + norm_about_one(feed_forward(w, p + "mlp.", norm_about_one(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
    return x


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence; `layers_out` receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    E = w["embed"].to(dtype)
    x = E[torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    first: Dict[str, torch.Tensor] = {}
    for i, l in enumerate(cfg["layers"]):
        x = layer(i, l, w, x, eps, first)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_about_one(x, w["final.norm"], eps) @ E.t() * float(cfg.get("logit_scale", 1.0))

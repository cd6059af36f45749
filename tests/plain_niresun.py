"""A plain, slow restatement of the Niresun decoder, one function per mechanism, on the CPU.

It shares no code with the package: tensors come in as a dict of torch tensors by name, the configuration as the
parsed config.json.  Everything is computed in the dtype asked for (float64 in the tests), one whole sequence at a
time, recurrences token by token.

Notation: x [n, W] is the residual stream of one sequence, positions 0..n-1.

    x_0 = E[token]
    layer:      x <- x + mixer(D(x; 1));   x <- x + ff(D(x; 2))         (ff may be absent)
    D(y):       tanh(alpha y) * w + b                                   no mean, no variance
    mixer:      a selective scan ("mamba1"), attention inside chunks of positions behind a gate ("attention"), or
                attention over everything beside a matrix memory ("parallel": half the sum of the two normed outputs)
    ff:         W_down (gelu_tanh(W_gate y) * W_up y)
    output:     logits = W_head D(x; final)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ----------------------------------------------------------------------------------------------- small pieces
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def dynamic_tanh(x: torch.Tensor, w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    d = x.dtype
    return torch.tanh(w[name + ".alpha"].to(d).reshape(()) * x) * w[name].to(d) + w[name + ".b"].to(d)


def linear(x: torch.Tensor, w: Dict[str, torch.Tensor], name: str, bias: bool = False) -> torch.Tensor:
    y = x @ w[name].to(x.dtype).t()
    return y + w[name + ".b"].to(x.dtype) if bias else y


def causal_conv(u: torch.Tensor, taps: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """u [n, C], taps [C, k]: y_t = sum_j taps[:, j] u_(t - k + 1 + j), zeros before the first row."""
    n, k = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(k):
        back = k - 1 - j
        if back < n:
            y[back:] += taps[:, j].to(u.dtype) * u[:n - back]
    return y if bias is None else y + bias.to(u.dtype)


# ----------------------------------------------------------------------------------------------- positions
def frequencies(rot: dict) -> torch.Tensor:
    dims, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for v in f.tolist():
        turns = original * v / (2.0 * math.pi)               # in `original` positions
        if turns > high:
            out.append(v)
        elif turns < low:
            out.append(v / factor)
        else:
            s = (turns - low) / (high - low) if high != low else 1.0
            out.append(v / factor + s * (v - v / factor))
    return torch.tensor(out, dtype=torch.float64)


def rotate_halves(v: torch.Tensor, rot: dict) -> torch.Tensor:
    """v [n, heads, d]: the pairs (i, i + dims / 2) of the first rot.dims elements turn by position * f_i."""
    half = int(rot["dims"]) // 2
    ang = torch.arange(v.shape[0], dtype=torch.float64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(ang).to(v.dtype)[:, None, :], torch.sin(ang).to(v.dtype)[:, None, :]
    a, b = v[..., :half], v[..., half:2 * half]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., 2 * half:]], dim=-1)


def query_temperature(n: int, coef: float, every: float) -> torch.Tensor:
    p = torch.arange(n, dtype=torch.float64)
    return 1.0 + coef * torch.log(torch.floor((p + 1.0) / every) + 1.0)


def unseen(n: int, dtype: torch.dtype, chunk: Optional[int] = None) -> torch.Tensor:
    """[n, n] with 0 where position i sees position j and -inf elsewhere: j <= i and, with chunks of positions counted
    from the sequence's start, only in i's own chunk."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    if chunk:
        see = see & (i // chunk == j // chunk)
    return torch.zeros(n, n, dtype=dtype).masked_fill(~see, -math.inf)


def softmax_attention(q, k, v, scale, mask):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H, dv]; query head h reads kv head h // (H // G)."""
    H, G = q.shape[1], k.shape[1]
    own = [h // (H // G) for h in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, own]) * scale + mask
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, dim=-1), v[:, own])


# ----------------------------------------------------------------------------------------------- mixers
def chunked_attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = linear(h, w, p + "q", True).reshape(n, H, d), linear(h, w, p + "k", True).reshape(n, G, d)
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"])
    v = linear(h, w, p + "v", True).reshape(n, G, dv)
    o = softmax_attention(q, k, v, m["scale"], unseen(n, h.dtype, m["mask"]["size"])).reshape(n, H * dv)
    return linear(o * sigmoid(linear(h, w, p + "g")), w, p + "o")


def conv_attention(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Projections, a short convolution of each, unit q and k, a temperature on q, no rotation."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(linear(h, w, p + x), w[p + x + ".conv"]) for x in "qkv")
    q, k = unit(q.reshape(n, H, d), eps), unit(k.reshape(n, G, d), eps)
    t = m["q_temp"]
    q = q * query_temperature(n, t["coef"], t["every"]).to(q.dtype)[:, None, None]
    o = softmax_attention(q, k, v.reshape(n, G, dv), m["scale"], unseen(n, h.dtype))
    return linear(o.reshape(n, H * dv), w, p + "o")


def memory_scan(q, k, v, i, f):
    """q, k [n, H, d], v [n, H, dv], log gates i, f [n, H] -> o [n, H, dv], with the running maximum m from 0."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    z = torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + add[:, None] * k[t]
        den = torch.maximum((z * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def matrix_memory(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    n, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = linear(h, w, p + "q").reshape(n, H, d) * d ** -0.5
    k = linear(h, w, p + "k").reshape(n, H, d)
    v = linear(h, w, p + "v").reshape(n, H, dv)
    i = cap * torch.tanh(linear(h, w, p + "i", True) / cap)
    f = -softplus(-cap * torch.tanh(linear(h, w, p + "f", True) / cap))
    o = unit(memory_scan(q, k, v, i, f), eps).reshape(n, H * dv)
    return linear(o * w[p + "norm"].to(h.dtype) * sigmoid(linear(h, w, p + "g")), w, p + "o")


def parallel(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    left = unit(conv_attention(m["left"], w, p + "left.", h, eps), eps) * w[p + "left.out"].to(h.dtype)
    right = unit(matrix_memory(m["right"], w, p + "right.", h, eps), eps) * w[p + "right.out"].to(h.dtype)
    return 0.5 * (left + right)


def selective_scan(x, dt, A, B, C, D):
    """x, dt [n, c], A [c, s], B, C [n, s], D [c] -> y [n, c]."""
    S = torch.zeros_like(A)
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out)


def mamba1(m: dict, w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    R, N, dt_ = m["dt_rank"], m["state"], h.dtype
    x, z = linear(h, w, p + "in").split(m["inner"], dim=1)
    x = silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    low, B, C = linear(x, w, p + "x").split([R, N, N], dim=1)
    dt = softplus(linear(low, w, p + "dt", True))
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"].to(dt_)), B, C, w[p + "D"].to(dt_))
    return linear(y * silu(z), w, p + "o")


# ----------------------------------------------------------------------------------------------- the rest
def feed_forward(w: Dict[str, torch.Tensor], p: str, h: torch.Tensor) -> torch.Tensor:
    return linear(gelu_tanh(linear(h, w, p + "gate")) * linear(h, w, p + "up"), w, p + "down")


def layer(i: int, l: dict, w: Dict[str, torch.Tensor], x: torch.Tensor, eps: float) -> torch.Tensor:
    p, m = f"l{i}.", l["mixer"]
    h = dynamic_tanh(x, w, p + "norm1")
    if l["type"] == "mamba1":
        y = mamba1(m, w, p + "mix.", h)
    elif l["type"] == "parallel":
        y = parallel(m, w, p + "mix.", h, eps)
    else:
        y = chunked_attention(m, w, p + "mix.", h)
    x = x + y
    if l["mlp"] is not None:
        x = x + feed_forward(w, p + "mlp.", dynamic_tanh(x, w, p + "norm2"))
    return x


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence; `layers_out` receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"].to(dtype)[torch.tensor(tokens)]
    for i, l in enumerate(cfg["layers"]):
        x = layer(i, l, w, x, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(dynamic_tanh(x, w, "final.norm"), w, "head")

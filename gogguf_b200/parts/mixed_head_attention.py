"""Attention whose heads' weights are mixed after the softmax ("talking heads"), with positions in the queries'
temperature instead of a rotation.

    q = W_q h + b_q [heads x head_dim],  k = W_k h + b_k [kv_heads x head_dim],  v = W_v h + b_v [kv_heads x value_dim]
    q at position p is multiplied by 1 + coef log(1 + floor((p + 1) / every))                   (query_temperature)
    v: each head's run divided by its root mean square over value_dim                            (unit_values)
    v <- v + mu (v0 - v), v0 being the values that the step's source layer made for the same token, mu a stored
        number                                                                                   (value_mix)
    s = cap tanh(scale q . k / cap),   p_h(i, j) = exp(s_j) / (one + sum_j exp(s_j))             (softcap, extra_one)
    o_h = sigmoid(W_g h)_h * sum_j ( sum_g T[h, g] p_g(i, j) ) v_j                               (talking, head_gate)
    y = W_o concat_h o + b_o

Query head h reads kv head h / (heads / kv_heads), its mixed weights that kv head's values.  The cache holds the keys
and the values as they enter the sums (normed, mixed).  `one` is 1 with `extra_one`, else 0.

Spec parameters: hidden_size, num_heads, num_kv_heads, head_dim, value_dim, scale, eps, bias (default False), softcap (0
or absent: none), query_temperature {coef, every} (absent: none), unit_values, value_mix (absent, "source": this layer's
values are the ones later layers mix in, "mix"), extra_one, talking (False: T is the identity, nothing stored),
head_gate, window (absent: none), names.

Temperature, scores, softmax, mixing and gate are float32 in both compute paths.  In the bfloat16 path head sizes of up
to 128 run on the tensor cores (prompts on tcgen05, short stretches and decode steps on mma.sync);
GOGGUF_B200_MIXED_HEAD_MMA=0 keeps the plain kernel, their twin.
"""
from __future__ import annotations

import math
import os
from typing import Dict

import torch

from ..cache.sequence_cache import KVRequest, KVView
from ..config.spec import PartSpec
from ..csrc import kernels as K
from ..weights.loader import TensorDecl
from .base import Linear, Runtime, StepContext
from .registry import register_mixer

PROMPT_FORM_MIN_TOKENS = 48      # steps whose longest stretch of new tokens has at least this many take the tcgen05 form
DECODE_FORM_MAX_TOKENS = 4       # ... and steps that bring at most this many to each sequence the form for few rows

FIRST_VALUES = "mixed_head_first_values"      # workspace: the source layer's values of the step's tokens


@register_mixer("mixed_head_attention")
class MixedHeadAttentionMixer:
    @classmethod
    def _names(cls, spec: PartSpec) -> Dict[str, str]:
        n = dict(q="q", k="k", v="v", o="o", talk="talk", gate="g", value_mix="vmix", bias=".b")
        n.update(spec.get("names") or {})
        return n

    @classmethod
    def _sizes(cls, spec: PartSpec):
        return (int(spec["hidden_size"]), int(spec["num_heads"]), int(spec["num_kv_heads"]), int(spec["head_dim"]),
                int(spec["value_dim"]))

    @classmethod
    def tensors(cls, spec: PartSpec) -> Dict[str, TensorDecl]:
        W, H, G, d, dv = cls._sizes(spec)
        n = cls._names(spec)
        t = {n["q"]: TensorDecl(shape=(H * d, W)), n["k"]: TensorDecl(shape=(G * d, W)),
             n["v"]: TensorDecl(shape=(G * dv, W)), n["o"]: TensorDecl(shape=(W, H * dv))}
        if spec.get("bias"):
            for key in ("q", "k", "v", "o"):
                t[n[key] + n["bias"]] = TensorDecl(shape=(t[n[key]].shape[0],), init="zeros_normal")
        if spec.get("talking"):
            t[n["talk"]] = TensorDecl(shape=(H, H), init="near_identity")
        if spec.get("head_gate"):
            t[n["gate"]] = TensorDecl(shape=(H, W))
        if spec.get("value_mix"):
            t[n["value_mix"]] = TensorDecl(shape=(), init="half")
        return t

    @classmethod
    def cache_request(cls, spec: PartSpec) -> KVRequest:
        _, _, G, d, dv = cls._sizes(spec)
        return KVRequest(num_kv_heads=G, head_dim=d, window=spec.get("window"), value_dim=None if dv == d else dv)

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], rt: Runtime):
        self.rt = rt
        self.hidden, self.H, self.G, self.d, self.dv = self._sizes(spec)
        H, G, d, dv = self.H, self.G, self.d, self.dv
        if H % G:
            raise ValueError(f"mixed_head_attention: {H} query heads are not a multiple of {G} kv heads")
        self.scale = float(spec.get("scale") or 1.0 / math.sqrt(d))
        self.eps = float(spec["eps"])
        self.cap = float(spec.get("softcap") or 0.0)
        qt = spec.get("query_temperature")
        self.coef, self.every = (float(qt["coef"]), float(qt["every"])) if qt else (0.0, 1.0)
        if not self.every > 0:
            raise ValueError("mixed_head_attention: query_temperature.every must be positive")
        self.unit = bool(spec.get("unit_values"))
        self.value_mix = spec.get("value_mix") or None
        if self.value_mix not in (None, "source", "mix"):
            raise ValueError(f"mixed_head_attention: value_mix={self.value_mix!r} is not known (source, mix)")
        self.one = bool(spec.get("extra_one"))
        self.window = int(spec.get("window") or 0)
        n = self._names(spec)
        gated = bool(spec.get("head_gate"))
        # rows of the first product: q heads, k heads, v heads, the heads' gate logits, filled up so that every
        # token's row starts on a 16-byte boundary
        keys = ["q", "k", "v"] + (["gate"] if gated else [])
        mats = [rt.matrix(weights[n[key]]) for key in keys]
        if len({m.dtype for m in mats}) != 1:
            mats = [m.float() for m in mats]
        rows = sum(m.shape[0] for m in mats)
        if rows % 8:
            mats.append(mats[0].new_zeros((8 - rows % 8, self.hidden)))
        w = torch.cat(mats, dim=0)
        bias = None
        if spec.get("bias"):
            parts = [rt.vector(weights[n[key] + n["bias"]]) for key in ("q", "k", "v")]
            bias = torch.cat(parts)
            bias = torch.cat([bias, bias.new_zeros(w.shape[0] - bias.numel())])
        self.proj = Linear(w, rt, bias=bias)
        self.k_off, self.v_off = H * d, (H + G) * d
        self.g_off = self.v_off + G * dv if gated else -1
        self.o = Linear(weights[n["o"]], rt, bias=weights[n["o"] + n["bias"]] if spec.get("bias") else None)
        self.talk = (rt.vector(weights[n["talk"]]) if spec.get("talking")
                     else torch.eye(H, dtype=torch.float32, device=rt.device))
        self.lam = float(weights[n["value_mix"]].double()) if self.value_mix == "mix" else 0.0
        self._mma = (rt.fast and rt.dtype == torch.bfloat16
                     and os.environ.get("GOGGUF_B200_MIXED_HEAD_MMA", "1") != "0")

    def absorb_norm(self, norm) -> bool:
        """Take the block's pre-norm into the first product; `forward` then gets RowStats as `h`."""
        if not self.proj.can_fold or norm.size != self.hidden:
            return False
        self.proj.fold_input_norm(norm.weight, norm.eps)
        return True

    def forward(self, h: torch.Tensor, residual: torch.Tensor, ctx: StepContext, cache: KVView,
                writes_cache: bool = True) -> None:
        if not writes_cache:
            raise ValueError("mixed_head_attention: the layer writes the keys and values that it reads")
        T, H, G, d, dv = ctx.n_tokens, self.H, self.G, self.d, self.dv
        row = ctx.ws.get("mixed_head_proj", (T, self.proj.out_features), self.rt.dtype)
        self.proj(h, row, ws=ctx.ws)
        table = ctx.page_tables[cache.group]
        first = keep = None
        if self.value_mix is not None:
            buf = ctx.ws.get(FIRST_VALUES, (T, G * dv), torch.float32)
            first, keep = (None, buf) if self.value_mix == "source" else (buf, None)
        K.head_kv_prep(row, self.k_off, self.v_off, cache.k, cache.v, ctx.positions, ctx.seq_of_token, table,
                       cache.page_size, T, G, d, dv, self.unit, self.eps, first, self.lam, keep)
        o = ctx.ws.get("mixed_head_out", (T, H * dv), self.rt.dtype)
        kw = dict(cap=self.cap, coef=self.coef, every=self.every, one=self.one, window=self.window)
        if (self._mma and ctx.max_new >= PROMPT_FORM_MIN_TOKENS
                and K.mixed_head_prompt_takes(H, G, d, dv, cache.page_size)):
            u = ctx.ws.get("mixed_head_u", (T * H * G * dv,), torch.float32)
            ml = ctx.ws.get("mixed_head_ml", (T * H * 2,), torch.float32)
            K.mixed_head_attention_prompt(row, self.g_off, cache.k, cache.v, o, self.talk, ctx.seq_of_token, ctx.cu_seqlens,
                                          ctx.ctx_lens, table, cache.page_size, T, ctx.n_seqs, H, G, d, dv, self.scale, u, ml, **kw)
        elif (self._mma and ctx.max_new <= DECODE_FORM_MAX_TOKENS
                and K.mixed_head_decode_takes(H, G, d, dv, cache.page_size)):
            nsplit = K.mixed_head_decode_splits(T, G, int(ctx.max_ctx))
            scores = ctx.ws.get("mixed_head_scores", (T, H, -(-int(ctx.max_ctx) // 64) * 64), torch.float32)
            ml = ctx.ws.get("mixed_head_ml", (T * H * nsplit * 2,), torch.float32)
            part = ctx.ws.get("mixed_head_part", (T * H * nsplit * dv,), torch.float32)
            K.mixed_head_attention_decode(row, self.g_off, cache.k, cache.v, o, self.talk, ctx.positions, ctx.seq_of_token, table,
                                          cache.page_size, T, H, G, d, dv, self.scale, scores, ml, part, nsplit, **kw)
        elif self._mma and K.mixed_head_mma_takes(H, G, d, dv, cache.page_size):
            # (steps of few rows over long contexts: the key tiles are shared out over several CTAs)
            nsplit = K.mixed_head_splits(T, ctx.n_seqs, H, G, int(ctx.max_ctx)) if ctx.max_new <= DECODE_FORM_MAX_TOKENS else 1
            u = ctx.ws.get("mixed_head_u", (T * H * nsplit * G * dv,), torch.float32)
            ml = ctx.ws.get("mixed_head_ml", (T * H * nsplit * 2,), torch.float32)
            K.mixed_head_attention_mma(row, self.g_off, cache.k, cache.v, o, self.talk, ctx.positions, ctx.seq_of_token,
                                       ctx.cu_seqlens, table, cache.page_size, T, ctx.n_seqs, H, G, d, dv, self.scale, u, ml,
                                       nsplit=nsplit, max_new=int(ctx.max_new), **kw)
        else:
            K.mixed_head_attention_plain(row, self.g_off, cache.k, cache.v, o, self.talk, ctx.positions, ctx.seq_of_token,
                                         table, cache.page_size, T, H, G, d, dv, self.scale, **kw)
        self.o(o, residual, accumulate=True, ws=ctx.ws)

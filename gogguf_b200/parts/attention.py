"""Grouped-query attention mixer with optional per-head q/k RMSNorm and a position encoding.

Order of operations as in the reference (pkg/model/qwen3/model.go:215-260): q, k, v projections
without bias; each q and k head normed over its `head_dim` slice with one shared weight (before the
rotation); rotation of q and k; k (normed, rotated) and v (raw) appended to the cache; attention of
every new token over the cached positions it may see; output projection added to the residual.
Score scale is 1/sqrt(head_dim) unless the spec gives `scale` (pkg/ops/attention.go:24).

Further parameters of the spec, each with the default that leaves the above unchanged: `value_dim` (head size of
v and of the attention output where it differs from `head_dim`), `qk_norm` = "whole" (q normed over its whole
projection with a weight of that size, k alike, instead of head by head), `sink` (a stored number per query head
that joins the softmax's denominator as exp(sink_h), without key, value or scale), `bias` (True: q, k and v have biases,
stored under their names with names["bias"] added), `taps` (a causal convolution over time of every column of q, k and v,
directly after the projections: y_t = sum_j c[:, j] u_(t - taps + 1 + j), zeros before the sequence's start, stored as
[columns, taps] under the projections' names with names["conv"] added; its last taps - 1 inputs are a state of the
sequence, and the part's cache request is then the pair of that and the keys and values), `qk_norm` = "unit" (q and k
divided by their root mean square head by head, no weight), `query_temperature` {coef, every} (q at position p is
multiplied by 1 + coef ln(1 + floor((p + 1) / every))), `position` None (no rotation), `chunk` (a position sees its own
chunk of that many positions only, counted from the sequence's start), `output_gate` (the concatenated heads are
multiplied element by element by sigmoid(W_g h)), `names` (the stored tensors' local names; keys q, k, v, o, q_norm, k_norm,
sink, gate, bias, conv).  `scale_output(m)` puts a factor on the attention output
in float32, before it is rounded for the output projection.
"""
from __future__ import annotations

import math
import os
from typing import Dict, Optional

import torch

from ..cache.sequence_cache import KVRequest, StateRequest
from ..config.spec import PartSpec
from ..csrc import kernels as K
from ..csrc import tcgen05_gemm
from ..weights.loader import TensorDecl
from .base import Linear, Runtime, StepContext
from .registry import POSITIONS, lookup, register_mixer

MAX_HEAD_DIM = 256


@register_mixer("attention")
class AttentionMixer:
    overwrites = True           # stores its output instead of adding it where ctx.shared["output_empty"] is set

    @classmethod
    def _names(cls, spec: PartSpec) -> Dict[str, str]:
        n = dict(q="q_proj.weight", k="k_proj.weight", v="v_proj.weight", o="o_proj.weight",
                 q_norm="q_norm.weight", k_norm="k_norm.weight", sink="sink", gate="g_proj.weight", bias=".b", conv=".conv")
        n.update(spec.get("names") or {})
        return n

    @classmethod
    def _norm_mode(cls, spec: PartSpec) -> int:
        """0: no q/k norm; 1: head by head; 2: over the whole projection.  ("unit": 1 without weights.)"""
        v = spec.get("qk_norm")
        if not v:
            return 0
        if v is True or v in ("head", "unit"):
            return 1
        if v == "whole":
            return 2
        raise ValueError(f"attention: qk_norm={v!r} is not known (False, True / 'head', 'whole', 'unit')")

    @classmethod
    def tensors(cls, spec: PartSpec) -> Dict[str, TensorDecl]:
        h, nq, nkv, d = spec["hidden_size"], spec["num_heads"], spec["num_kv_heads"], spec["head_dim"]
        dv = spec.get("value_dim") or d
        n = cls._names(spec)
        t = {
            n["q"]: TensorDecl(shape=(nq * d, h)),
            n["k"]: TensorDecl(shape=(nkv * d, h)),
            n["v"]: TensorDecl(shape=(nkv * dv, h)),
            n["o"]: TensorDecl(shape=(h, nq * dv)),
        }
        mode = cls._norm_mode(spec)
        if mode and spec.get("qk_norm") != "unit":
            t[n["q_norm"]] = TensorDecl(shape=(d if mode == 1 else nq * d,), init="ones_normal")
            t[n["k_norm"]] = TensorDecl(shape=(d if mode == 1 else nkv * d,), init="ones_normal")
        if spec.get("sink"):
            t[n["sink"]] = TensorDecl(shape=(nq,), init="small_normal")
        if spec.get("output_gate"):
            t[n["gate"]] = TensorDecl(shape=(nq * dv, h))
        for key in ("q", "k", "v"):
            rows = t[n[key]].shape[0]
            if spec.get("bias"):
                t[n[key] + n["bias"]] = TensorDecl(shape=(rows,), init="zeros_normal")
            if spec.get("taps"):
                t[n[key] + n["conv"]] = TensorDecl(shape=(rows, int(spec["taps"])), init="small_normal")
        return t

    @classmethod
    def cache_request(cls, spec: PartSpec):
        nq, nkv, d = int(spec["num_heads"]), int(spec["num_kv_heads"]), int(spec["head_dim"])
        dv = int(spec.get("value_dim") or d)
        kv = KVRequest(num_kv_heads=nkv, head_dim=d, window=spec.get("window"), value_dim=None if dv == d else dv,
                       chunk=spec.get("chunk"))
        taps = int(spec.get("taps") or 0)
        if taps <= 1:                       # (no convolution, or one that keeps nothing)
            return kv
        return (StateRequest(shape=(taps - 1, nq * d + nkv * (d + dv)), dtype=torch.float32), kv)

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], rt: Runtime):
        self.rt = rt
        self.hidden = int(spec["hidden_size"])
        self.nq = int(spec["num_heads"])
        self.nkv = int(spec["num_kv_heads"])
        self.d = int(spec["head_dim"])
        self.dv = int(spec.get("value_dim") or self.d)
        if self.nq % self.nkv:
            raise ValueError(f"attention: {self.nq} query heads are not a multiple of {self.nkv} kv heads")
        if self.d > MAX_HEAD_DIM:
            raise ValueError(f"attention: head_dim={self.d} is not supported (at most {MAX_HEAD_DIM})")
        if self.dv > MAX_HEAD_DIM:
            raise ValueError(f"attention: value_dim={self.dv} is not supported (at most {MAX_HEAD_DIM})")
        self.window = int(spec.get("window") or 0)
        self.scale = float(spec.get("scale") or 1.0 / math.sqrt(self.d))
        self.eps = float(spec.get("qk_norm_eps", 0.0))
        self.chunk = int(spec.get("chunk") or 0)
        pos = dict(spec["position"]) if spec.get("position") is not None else None
        self.position = lookup(POSITIONS, pos["kind"], "position encoding")(pos, rt) if pos is not None else None
        self.rot = int(pos.get("rotary_dim", self.d)) if pos is not None else 0
        qt = spec.get("query_temperature")
        self.coef, self.every = (float(qt["coef"]), float(qt["every"])) if qt else (0.0, 1.0)
        if not self.every > 0:
            raise ValueError("attention: query_temperature.every must be positive")
        if self.rot > self.d:
            raise ValueError("attention: rotary_dim exceeds head_dim")
        names = self._names(spec)
        self.gated = bool(spec.get("output_gate"))
        mats = [rt.matrix(weights[names[n]]) for n in ("q", "k", "v") + (("gate",) if self.gated else ())]
        if len({m.dtype for m in mats}) != 1:
            mats = [m.float() for m in mats]
        # rows: all q heads, then all k heads, then all v heads, then (gated) the gate's logits, which start, like every
        # token's row, on a 16-byte boundary
        self.cols = self.nq * self.d + self.nkv * (self.d + self.dv)
        self.g_off = -(-self.cols // 8) * 8 if self.gated else 0
        if self.gated:
            fill = [mats[0].new_zeros((n, self.hidden)) for n in (self.g_off - self.cols, -(self.g_off + self.nq * self.dv) % 8)]
            mats = mats[:3] + [f for f in fill[:1] if f.shape[0]] + mats[3:] + [f for f in fill[1:] if f.shape[0]]
        w = torch.cat(mats, dim=0)
        bias = None
        if spec.get("bias"):
            bias = torch.cat([rt.vector(weights[names[n] + names["bias"]]) for n in ("q", "k", "v")])
            bias = torch.cat([bias, bias.new_zeros(w.shape[0] - bias.numel())])
        self.qkv = Linear(w, rt, bias=bias)
        self.taps = int(spec.get("taps") or 0)
        # [taps, columns]: a tap's weights side by side
        self.conv = (torch.cat([rt.vector(weights[names[n] + names["conv"]]) for n in ("q", "k", "v")]).t().contiguous()
                     if self.taps else None)
        self.o = Linear(weights[names["o"]], rt)
        self.norm_mode = self._norm_mode(spec)
        if self.norm_mode and spec.get("qk_norm") != "unit":
            self.q_norm = rt.vector(weights[names["q_norm"]])
            self.k_norm = rt.vector(weights[names["k_norm"]])
        else:
            self.q_norm = self.k_norm = None
        self.sink = rt.vector(weights[names["sink"]]) if spec.get("sink") else None
        self.out_scale = 1.0
        # what the kernels written for one head size, a norm head by head and a plain softmax do not take
        self._general = (self.dv != self.d or self.norm_mode == 2 or bias is not None or self.conv is not None or self.gated
                         or spec.get("qk_norm") == "unit" or qt is not None or self.position is None or self.d % 2 != 0)
        self._fast = None
        if rt.fast and rt.dtype == torch.bfloat16:
            from ..csrc import fast_attention
            self._fast = fast_attention.try_make(self.nq, self.nkv, self.d, self.scale, self.window, dv=self.dv, chunk=self.chunk)
        # head size 128 with a full rotation by cos/sin tables: the decode form of the q/k/v product can do
        # the per-head work itself (one head per 128-row weight tile)
        self._fused_rope = (self.qkv.tensor_core and self.d == 128 and self.rot == self.d and not self._general
                            and os.environ.get("GOGGUF_B200_FUSE_QKV_ROPE", "1") != "0")

    def can_absorb_norm(self, norm) -> bool:
        return self.qkv.can_fold and norm.size == self.hidden

    def absorb_norm(self, norm) -> bool:
        """Take the block's pre-norm into the q/k/v projection; `forward` then gets RowStats as `h`."""
        if not self.can_absorb_norm(norm):
            return False
        self.qkv.fold_input_norm(norm.weight, norm.eps)
        return True

    def scale_output(self, mult: float) -> bool:
        """A factor on this mixer's output: the attention kernels apply it to their float32 result."""
        self.out_scale = float(mult)
        return True

    def prepare(self, ctx: StepContext) -> None:
        if self.position is not None:
            self.position.tables(ctx)

    def forward(self, h: torch.Tensor, residual: torch.Tensor, ctx: StepContext, cache, writes_cache: bool = True) -> None:
        tail = None
        if self.taps > 1:
            tail, cache = cache
        if self.taps and not writes_cache:
            raise ValueError("attention: a layer's convolution state cannot be read by another layer")
        T, nq, nkv, d, dv = ctx.n_tokens, self.nq, self.nkv, self.d, self.dv
        dt = self.rt.dtype
        q = ctx.ws.get("attn_q", (T, nq * d), dt)
        o = ctx.ws.get("attn_out", (T, nq * dv), dt)
        cos, sin = self.position.tables(ctx) if self.position is not None else (None, None)
        table = ctx.page_tables[cache.group]
        gate = None
        if self._fused_rope and tcgen05_gemm.qkv_rope_takes(T):
            # norm, rotation and cache write happen in the projection's epilogue
            self.qkv.qkv_rope(h, T, ws=ctx.ws, q_out=q, qw=self.q_norm, kw=self.k_norm, eps=self.eps, cos=cos, sin=sin,
                              positions=ctx.positions, seq_of_token=ctx.seq_of_token, page_table=table,
                              page_size=cache.page_size, k_pool=cache.k if writes_cache else None,
                              v_pool=cache.v if writes_cache else None, nq=nq, nkv=nkv)
        elif self._general:
            row = ctx.ws.get("attn_qkv", (T, self.qkv.out_features), dt)
            self.qkv(h, row, ws=ctx.ws)
            if self.gated:
                gate = row[:, self.g_off:self.g_off + nq * dv]
            K.qkv_prep(row[:, :self.cols], q, self.q_norm, self.k_norm, self.eps, self.norm_mode, cos, sin, ctx.positions,
                       ctx.seq_of_token, table, cache.page_size, cache.k if writes_cache else None,
                       cache.v if writes_cache else None, T, nq, nkv, d, dv, self.rot, conv=self.conv,
                       conv_state=tail.state if tail is not None else None, cu_seqlens=ctx.cu_seqlens, slots=ctx.slots,
                       n_seqs=ctx.n_seqs, max_new=int(ctx.max_new), coef=self.coef, every=self.every)
        else:
            qkv = ctx.ws.get("attn_qkv", (T, (nq + 2 * nkv) * d), dt)
            self.qkv(h, qkv, ws=ctx.ws)
            K.qk_norm_rope_cache(qkv, q, self.q_norm, self.k_norm, self.eps, cos, sin, ctx.positions,
                                 ctx.seq_of_token, table, cache.page_size,
                                 cache.k if writes_cache else None, cache.v if writes_cache else None,
                                 T, nq, nkv, d, self.rot)
        if self._fast is not None:
            self._fast(q, cache.k, cache.v, o, ctx, table, cache.page_size, sink=self.sink, out_scale=self.out_scale, gate=gate)
        else:
            K.attention_plain(q, cache.k, cache.v, o, ctx.positions, ctx.seq_of_token, table,
                              cache.page_size, T, nq, nkv, d, self.scale, self.window, dv=dv, sink=self.sink,
                              out_scale=self.out_scale, chunk=self.chunk, gate=gate)
        self.o(o, residual, accumulate=not ctx.shared.get("output_empty", False), ws=ctx.ws, emit=ctx.shared.get("row_stats"))

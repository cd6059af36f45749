"""Typed configuration of the Kulesun decoder, read from its config.json keys.

A Kulesun model is a list of layers that may differ from one another.  The embedding is multiplied by a factor.  A
layer has a norm before and after each of its two parts (weights stored as their distance from one):

    x += N1b(mixer(N1(x)));   x += N2b(ff(N2(x)))        (the feed-forward may be absent)

The mixer is latent attention (an uncompressed query with a rotated part in halves and stretched frequencies, one
rotated key part for all heads, a gate on every element of the heads' outputs) or attention without a rotation
(biases, a query temperature that grows with the position, values of unit root mean square mixed with those of the
first such layer, bounded scores, one in the softmax's denominator, the heads' weights mixed by a stored matrix, a gate
per head).  The feed-forward is W_down (silu(W_gate x) * W_up x).  The head is the embedding table (without its
factor), the logits are multiplied by a factor.

config.json keys (every size and constant comes from here):

    architecture     "Kulesun"
    vocab, width     vocabulary and width of the residual stream
    norm.eps         epsilon of every RMS norm
    embedding.scale  factor on the embedded rows (default 1)
    logit_scale      factor on the logits (default 1)
    layers[i]        type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, scale,
                                                     rot {base, dims, scaling {factor, original, fast, slow}}}
                     type "attention":        mixer {heads, kv_heads, dim, vdim, scale, softcap, v_mix,
                                                     q_temp {coef, every}}
                     mlp null | {kind "dense", ff}

Tensor names: ``embed``, ``final.norm`` and per layer i ``l<i>.norm{1,1b,2,2b}``;
``l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}`` or ``l<i>.mix.{q,q.b,k,k.b,v,v.b,vmix,talk,g,o,o.b}``;
``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .registry import ConfigError, register_architecture
from .spec import BlockSpec, ModelSpec, PartSpec, default_schedule

# the positions have no trained limit that the design enforces: the cache bounds a sequence
MAX_POSITIONS = 1 << 22

MIXER_TYPES = ("latent_attention", "attention")
SCALING_KEYS = ("factor", "original", "fast", "slow")


def _need(d: Any, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"kulesun config: {where} needs {key!r}")
    return d[key]


def _pos_int(d: Any, key: str, where: str) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"kulesun config: {where}.{key} must be a positive integer, got {v!r}")
    return v


def _number(d: Any, key: str, where: str) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"kulesun config: {where}.{key} must be a number, got {v!r}")
    return float(v)


def _optional_number(d: Any, key: str, where: str, default: float) -> float:
    return default if not isinstance(d, dict) or d.get(key) is None else _number(d, key, where)


@dataclass(frozen=True)
class MixerConfig:
    heads: int
    dim: int
    vdim: int
    scale: float
    # latent attention
    rot_dim: int = 0
    kv_rank: int = 0
    rot_base: float = 0.0
    rot_dims: int = 0
    rot_scaling: Optional[Tuple[float, float, float, float]] = None      # factor, original, fast, slow
    # attention
    kv_heads: int = 0
    softcap: float = 0.0
    v_mix: bool = False
    q_temp: Optional[Tuple[float, float]] = None                         # coef, every

    @classmethod
    def from_dict(cls, kind: str, d: Any, where: str) -> "MixerConfig":
        base = dict(heads=_pos_int(d, "heads", where), dim=_pos_int(d, "dim", where), vdim=_pos_int(d, "vdim", where),
                    scale=_number(d, "scale", where))
        if kind == "latent_attention":
            rot_dim = d.get("rot_dim") or 0
            if isinstance(rot_dim, bool) or not isinstance(rot_dim, int) or rot_dim < 0:
                raise ConfigError(f"kulesun config: {where}.rot_dim must be a count, got {rot_dim!r}")
            base.update(rot_dim=rot_dim, kv_rank=_pos_int(d, "kv_rank", where))
            if rot_dim:
                rot = _need(d, "rot", where)
                dims = rot_dim if rot.get("dims") is None else rot["dims"]
                if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > rot_dim:
                    raise ConfigError(f"kulesun config: {where}.rot.dims must be even and at most rot_dim={rot_dim}, got {dims!r}")
                rb = _number(rot, "base", where + ".rot")
                if not rb > 1.0:
                    raise ConfigError(f"kulesun config: {where}.rot.base must be above one, got {rb}")
                sc = rot.get("scaling")
                base.update(rot_dims=dims, rot_base=rb, rot_scaling=None if sc is None else tuple(
                    _number(sc, k, where + ".rot.scaling") for k in SCALING_KEYS))
            return cls(**base)
        kv = _pos_int(d, "kv_heads", where)
        if base["heads"] % kv:
            raise ConfigError(f"kulesun config: {where}: {base['heads']} heads are not a multiple of {kv} kv_heads")
        cap = _optional_number(d, "softcap", where, 0.0)
        if cap < 0:
            raise ConfigError(f"kulesun config: {where}.softcap must not be negative, got {cap}")
        v_mix = d.get("v_mix", False)
        if v_mix is not None and not isinstance(v_mix, bool):
            raise ConfigError(f"kulesun config: {where}.v_mix must be true or false, got {v_mix!r}")
        qt = d.get("q_temp")
        temp = None
        if qt is not None:
            temp = (_number(qt, "coef", where + ".q_temp"), _number(qt, "every", where + ".q_temp"))
            if not temp[1] > 0:
                raise ConfigError(f"kulesun config: {where}.q_temp.every must be positive, got {temp[1]}")
        return cls(kv_heads=kv, softcap=cap, v_mix=bool(v_mix), q_temp=temp, **base)

    def to_dict(self, kind: str) -> Dict[str, Any]:
        d: Dict[str, Any] = dict(heads=self.heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if kind == "latent_attention":
            d.update(rot_dim=self.rot_dim, kv_rank=self.kv_rank)
            if self.rot_dim:
                d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
                if self.rot_scaling is not None:
                    d["rot"]["scaling"] = dict(zip(SCALING_KEYS, self.rot_scaling))
            return d
        d.update(kv_heads=self.kv_heads, v_mix=self.v_mix)
        if self.softcap:
            d["softcap"] = self.softcap
        if self.q_temp is not None:
            d["q_temp"] = dict(coef=self.q_temp[0], every=self.q_temp[1])
        return d


@dataclass(frozen=True)
class KulesunLayer:
    type: str
    mixer: MixerConfig
    ff: int                     # 0: no feed-forward


@register_architecture("Kulesun", "kulesun")
@dataclass(frozen=True)
class KulesunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[KulesunLayer, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "KulesunConfig":
        raw = _need(d, "layers", "config")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("kulesun config: 'layers' must be a non-empty list")
        layers: List[KulesunLayer] = []
        source: Optional[MixerConfig] = None       # the first layer whose values later ones mix in
        for i, ld in enumerate(raw):
            where = f"layers[{i}]"
            kind = _need(ld, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"kulesun config: {where}.type={kind!r} is not known ({', '.join(MIXER_TYPES)})")
            mixer = MixerConfig.from_dict(kind, _need(ld, "mixer", where), where + ".mixer")
            if mixer.v_mix:
                if source is None:
                    source = mixer
                elif (mixer.kv_heads, mixer.vdim) != (source.kv_heads, source.vdim):
                    raise ConfigError(f"kulesun config: {where}.mixer mixes in the first v_mix layer's values; kv_heads and "
                                      "vdim must equal that layer's")
            mlp = ld.get("mlp")
            ff = 0
            if mlp is not None:
                mk = _need(mlp, "kind", where + ".mlp")
                if mk != "dense":
                    raise ConfigError(f"kulesun config: {where}.mlp.kind={mk!r} is not known (dense)")
                ff = _pos_int(mlp, "ff", where + ".mlp")
            layers.append(KulesunLayer(type=kind, mixer=mixer, ff=ff))
        eps = _number(_need(d, "norm", "config"), "eps", "norm")
        if not eps > 0:
            raise ConfigError(f"kulesun config: norm.eps must be > 0, got {eps}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(x) for x in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"), norm_eps=eps,
                   layers=tuple(layers), embedding_scale=_optional_number(d.get("embedding"), "scale", "embedding", 1.0),
                   logit_scale=_optional_number(d, "logit_scale", "config", 1.0), eos_token_ids=eos_ids,
                   initializer_range=float(d.get("initializer_range", 0.05)))

    # ------------------------------------------------------------------ write
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": "Kulesun", "vocab": self.vocab, "width": self.width,
                             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                             "logit_scale": self.logit_scale,
                             "layers": [{"type": l.type, "mixer": l.mixer.to_dict(l.type),
                                         "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None} for l in self.layers]}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids) if len(self.eos_token_ids) > 1 else self.eos_token_ids[0]
        return d

    # ------------------------------------------------------------- derived
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def parameter_count(self) -> int:
        W = self.width
        n = self.vocab * W + W
        for l in self.layers:
            m = l.mixer
            n += 2 * W
            if l.type == "latent_attention":
                n += m.heads * (m.dim + m.rot_dim) * W + (m.kv_rank + m.rot_dim) * W + m.kv_rank
                n += m.heads * (m.dim + m.vdim) * m.kv_rank + 2 * m.heads * m.vdim * W
            else:
                rows = m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)
                n += rows * (W + 1) + m.heads * W + m.heads * m.heads + m.heads * m.vdim * W + W + int(m.v_mix)
            if l.ff:
                n += 2 * W + 3 * l.ff * W
        return n

    def kv_bytes_per_token(self, itemsize: int = 2) -> int:
        """Bytes a token adds to the paged caches."""
        return sum((l.mixer.kv_rank + l.mixer.rot_dim if l.type == "latent_attention"
                    else l.mixer.kv_heads * (l.mixer.dim + l.mixer.vdim)) * itemsize for l in self.layers)

    # ---------------------------------------------------------------- spec
    def _mixer(self, l: KulesunLayer, p: str, value_mix: Optional[str]) -> PartSpec:
        W, eps, m = self.width, self.norm_eps, l.mixer
        if l.type == "latent_attention":
            position = None
            if m.rot_dim:
                position = dict(kind="rope_neox", theta=m.rot_base, rotary_dim=m.rot_dims)
                if m.rot_scaling is not None:
                    position.update(kind="rope_yarn", **dict(zip(SCALING_KEYS, m.rot_scaling)))
            return PartSpec(kind="latent_attention", prefix=p, params=dict(
                hidden_size=W, num_heads=m.heads, nope_dim=m.dim, rope_dim=m.rot_dim, value_dim=m.vdim, latent_dim=m.kv_rank,
                scale=m.scale, window=None, latent_norm_eps=eps, position=position, output_gate=True,
                names=dict(q="q", down="dkv", latent_norm="dkv.norm", up_k="uk", up_v="uv", gate="g", out="o")))
        return PartSpec(kind="mixed_head_attention", prefix=p, params=dict(
            hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
            bias=True, softcap=m.softcap, query_temperature=None if m.q_temp is None else dict(zip(("coef", "every"), m.q_temp)),
            unit_values=True, value_mix=value_mix, extra_one=True, talking=True, head_gate=True))

    def to_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        blocks: List[BlockSpec] = []
        have_source = False

        def norm(p: str, name: str) -> PartSpec:
            return PartSpec(kind="rmsnorm", prefix=p, params=dict(size=W, eps=eps, tensor=name, weight_offset=1.0))

        for i, l in enumerate(self.layers):
            p = f"l{i}."
            value_mix = None
            if l.mixer.v_mix:
                value_mix = "mix" if have_source else "source"
                have_source = True
            parts: Dict[str, PartSpec] = {"mixer": self._mixer(l, p + "mix.", value_mix), "mixer_norm": norm(p, "norm1"),
                                          "mixer_post_norm": norm(p, "norm1b")}
            if l.ff:
                parts.update(feed_forward=PartSpec(kind="swiglu", prefix=p + "mlp.", params=dict(
                    hidden_size=W, intermediate_size=l.ff, names=dict(gate="gate", up="up", down="down"))),
                    feed_forward_norm=norm(p, "norm2"), feed_forward_post_norm=norm(p, "norm2b"))
            blocks.append(BlockSpec("sandwich_norm", parts))
        spec = ModelSpec(
            architecture="Kulesun", vocab_size=self.vocab, hidden_size=W, max_positions=MAX_POSITIONS,
            blocks=tuple(blocks), schedule=default_schedule(len(blocks)),
            embedding=PartSpec(kind="embedding", prefix="", params=dict(vocab_size=self.vocab, hidden_size=W,
                                                                        tensor="embed", scale=self.embedding_scale)),
            final_norm=PartSpec(kind="rmsnorm", prefix="final.", params=dict(size=W, eps=eps, tensor="norm", weight_offset=1.0)),
            head=PartSpec(kind="linear_head", prefix="", params=dict(vocab_size=self.vocab, hidden_size=W, tied_to="embed",
                                                                     tensor="head", scale=self.logit_scale)),
            stop_token_ids=self.eos_token_ids,
        )
        spec.validate()
        return spec

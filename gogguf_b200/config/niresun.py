"""Typed configuration of the Niresun decoder, read from its config.json keys.

A Niresun model is a list of layers that may differ from one another, each with a norm before its two parts:

    x += mixer(D(x));   x += ff(D(x))        (the feed-forward may be absent)      D(y) = tanh(alpha y) * w + b

The mixer is a selective scan (`mamba1`), softmax attention inside chunks of positions (biases, a partial rotation with
banded frequencies, a gate on every element of the heads' outputs), or two mixers side by side on the same input, half
the sum of whose normed outputs is added: attention over all positions without a rotation (a short convolution of q, k
and v, unit q and k, a query temperature that grows with the position) and a matrix memory with exponential gates.  The
feed-forward is W_down (gelu_tanh(W_gate x) * W_up x).  The head is a matrix of its own.

config.json keys (every size and constant comes from here):

    architecture     "Niresun"
    vocab, width     vocabulary and width of the residual stream
    norm.eps         epsilon of every RMS norm inside the mixers
    layers[i]        type "mamba1":    mixer {inner, state, dt_rank, conv}
                     type "attention": mixer {heads, kv_heads, dim, vdim, scale, mask {size},
                                              rot {base, dims, scaling {factor, low, high, original}}}
                     type "parallel":  mixer {left  {heads, kv_heads, dim, vdim, scale, conv, q_temp {coef, every}},
                                              right {heads, dim, vdim, gate_cap}}
                     mlp null | {kind "dense", ff}

Tensor names: ``embed``, ``head``, ``final.norm{,.alpha,.b}`` and per layer i ``l<i>.norm{1,2}{,.alpha,.b}``;
``l<i>.mix.{in,conv,conv.b,x,dt,dt.b,A_log,D,o}``, ``l<i>.mix.{q,q.b,k,k.b,v,v.b,g,o}`` or
``l<i>.mix.left.{q,k,v,q.conv,k.conv,v.conv,o,out}`` with ``l<i>.mix.right.{q,k,v,g,i,i.b,f,f.b,norm,o,out}``;
``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .registry import ConfigError, register_architecture
from .spec import BlockSpec, ModelSpec, PartSpec, default_schedule

# the positions have no trained limit that the design enforces: the cache bounds a sequence
MAX_POSITIONS = 1 << 22

MIXER_TYPES = ("mamba1", "attention", "parallel")
SCALING_KEYS = ("factor", "low", "high", "original")


def _need(d: Any, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"niresun config: {where} needs {key!r}")
    return d[key]


def _pos_int(d: Any, key: str, where: str) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"niresun config: {where}.{key} must be a positive integer, got {v!r}")
    return v


def _number(d: Any, key: str, where: str) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"niresun config: {where}.{key} must be a number, got {v!r}")
    return float(v)


def _optional_pos_int(d: Any, key: str, where: str) -> Optional[int]:
    return None if not isinstance(d, dict) or d.get(key) is None else _pos_int(d, key, where)


@dataclass(frozen=True)
class ScanConfig:
    """The selective scan."""
    inner: int
    state: int
    dt_rank: int
    conv: int

    @classmethod
    def from_dict(cls, d: Any, where: str) -> "ScanConfig":
        return cls(**{k: _pos_int(d, k, where) for k in ("inner", "state", "dt_rank", "conv")})

    def to_dict(self) -> Dict[str, Any]:
        return dict(inner=self.inner, state=self.state, dt_rank=self.dt_rank, conv=self.conv)


@dataclass(frozen=True)
class AttentionConfig:
    """Softmax attention: inside chunks with a rotation, or over everything behind a short convolution."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int] = None
    rot_dims: int = 0                                                    # 0: no rotation
    rot_base: float = 0.0
    rot_scaling: Optional[Tuple[float, float, float, float]] = None      # factor, low, high, original
    conv: Optional[int] = None
    q_temp: Optional[Tuple[float, float]] = None                         # coef, every

    @classmethod
    def _base(cls, d: Any, where: str) -> Dict[str, Any]:
        base = dict(heads=_pos_int(d, "heads", where), kv_heads=_pos_int(d, "kv_heads", where), dim=_pos_int(d, "dim", where),
                    vdim=_pos_int(d, "vdim", where), scale=_number(d, "scale", where))
        if base["heads"] % base["kv_heads"]:
            raise ConfigError(f"niresun config: {where}: {base['heads']} heads are not a multiple of {base['kv_heads']} kv_heads")
        return base

    @classmethod
    def chunked(cls, d: Any, where: str) -> "AttentionConfig":
        base = cls._base(d, where)
        base["chunk"] = _pos_int(_need(d, "mask", where), "size", where + ".mask")
        rot = d.get("rot")
        if rot is not None:
            dims = _need(rot, "dims", where + ".rot")
            if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > base["dim"]:
                raise ConfigError(f"niresun config: {where}.rot.dims must be even and at most dim={base['dim']}, got {dims!r}")
            b = _number(rot, "base", where + ".rot")
            if not b > 0:
                raise ConfigError(f"niresun config: {where}.rot.base must be positive, got {b}")
            base.update(rot_dims=dims, rot_base=b)
            sc = rot.get("scaling")
            if sc is not None:
                vals = tuple(_number(sc, k, where + ".rot.scaling") for k in SCALING_KEYS)
                if not all(v > 0 for v in vals):
                    raise ConfigError(f"niresun config: {where}.rot.scaling: {', '.join(SCALING_KEYS)} must be positive")
                base["rot_scaling"] = vals
        return cls(**base)

    @classmethod
    def convolved(cls, d: Any, where: str) -> "AttentionConfig":
        base = cls._base(d, where)
        base["conv"] = _optional_pos_int(d, "conv", where)
        qt = d.get("q_temp")
        if qt is not None:
            base["q_temp"] = (_number(qt, "coef", where + ".q_temp"), _number(qt, "every", where + ".q_temp"))
            if not base["q_temp"][1] > 0:
                raise ConfigError(f"niresun config: {where}.q_temp.every must be positive, got {base['q_temp'][1]}")
        return cls(**base)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.chunk is not None:
            d["mask"] = dict(size=self.chunk)
            if self.rot_base:
                d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
                if self.rot_scaling is not None:
                    d["rot"]["scaling"] = dict(zip(SCALING_KEYS, self.rot_scaling))
            return d
        if self.conv is not None:
            d["conv"] = self.conv
        if self.q_temp is not None:
            d["q_temp"] = dict(coef=self.q_temp[0], every=self.q_temp[1])
        return d


@dataclass(frozen=True)
class MemoryConfig:
    """The matrix memory."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: Any, where: str) -> "MemoryConfig":
        cap = _number(d, "gate_cap", where)
        if not cap > 0:
            raise ConfigError(f"niresun config: {where}.gate_cap must be positive, got {cap}")
        return cls(heads=_pos_int(d, "heads", where), dim=_pos_int(d, "dim", where), vdim=_pos_int(d, "vdim", where), gate_cap=cap)

    def to_dict(self) -> Dict[str, Any]:
        return dict(heads=self.heads, dim=self.dim, vdim=self.vdim, gate_cap=self.gate_cap)


@dataclass(frozen=True)
class PairConfig:
    left: AttentionConfig
    right: MemoryConfig

    @classmethod
    def from_dict(cls, d: Any, where: str) -> "PairConfig":
        return cls(left=AttentionConfig.convolved(_need(d, "left", where), where + ".left"),
                   right=MemoryConfig.from_dict(_need(d, "right", where), where + ".right"))

    def to_dict(self) -> Dict[str, Any]:
        return dict(left=self.left.to_dict(), right=self.right.to_dict())


_MIXER_READERS = {"mamba1": ScanConfig.from_dict, "attention": AttentionConfig.chunked, "parallel": PairConfig.from_dict}


@dataclass(frozen=True)
class NiresunLayer:
    type: str
    mixer: Any                  # ScanConfig, AttentionConfig or PairConfig
    ff: int                     # 0: no feed-forward


@register_architecture("Niresun", "niresun")
@dataclass(frozen=True)
class NiresunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[NiresunLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()
    initializer_range: float = 0.05

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NiresunConfig":
        raw = _need(d, "layers", "config")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("niresun config: 'layers' must be a non-empty list")
        layers: List[NiresunLayer] = []
        for i, ld in enumerate(raw):
            where = f"layers[{i}]"
            kind = _need(ld, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"niresun config: {where}.type={kind!r} is not known ({', '.join(MIXER_TYPES)})")
            mixer = _MIXER_READERS[kind](_need(ld, "mixer", where), where + ".mixer")
            mlp = ld.get("mlp")
            ff = 0
            if mlp is not None:
                mk = _need(mlp, "kind", where + ".mlp")
                if mk != "dense":
                    raise ConfigError(f"niresun config: {where}.mlp.kind={mk!r} is not known (dense)")
                ff = _pos_int(mlp, "ff", where + ".mlp")
            layers.append(NiresunLayer(type=kind, mixer=mixer, ff=ff))
        eps = _number(_need(d, "norm", "config"), "eps", "norm")
        if not eps > 0:
            raise ConfigError(f"niresun config: norm.eps must be > 0, got {eps}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(x) for x in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"), norm_eps=eps,
                   layers=tuple(layers), eos_token_ids=eos_ids, initializer_range=float(d.get("initializer_range", 0.05)))

    # ------------------------------------------------------------------ write
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": "Niresun", "vocab": self.vocab, "width": self.width,
                             "norm": {"eps": self.norm_eps},
                             "layers": [{"type": l.type, "mixer": l.mixer.to_dict(),
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

    def _attentions(self) -> List[AttentionConfig]:
        return [l.mixer.left if l.type == "parallel" else l.mixer for l in self.layers if l.type != "mamba1"]

    def parameter_count(self) -> int:
        W = self.width
        n = 2 * self.vocab * W + 2 * W + 1
        for l in self.layers:
            n += (2 * W + 1) * (2 if l.ff else 1) + 3 * l.ff * W
            if l.type == "mamba1":
                m = l.mixer
                n += 2 * m.inner * W + m.inner * (m.conv + 1) + (m.dt_rank + 2 * m.state) * m.inner
                n += m.inner * (m.dt_rank + 1) + m.inner * m.state + m.inner + W * m.inner
                continue
            a = l.mixer.left if l.type == "parallel" else l.mixer
            rows = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)
            n += rows * W + a.heads * a.vdim * W
            if l.type == "attention":
                n += rows + a.heads * a.vdim * W
            else:
                r = l.mixer.right
                n += rows * (a.conv or 0) + 2 * W
                n += 2 * r.heads * r.dim * W + 3 * r.heads * r.vdim * W + r.heads * r.vdim + 2 * r.heads * (W + 1)
        return n

    def kv_bytes_per_token(self, itemsize: int = 2) -> int:
        """Bytes a token adds to the paged caches (chunked layers give theirs back as chunks end)."""
        return sum(a.kv_heads * (a.dim + a.vdim) * itemsize for a in self._attentions())

    # ---------------------------------------------------------------- spec
    def _attention(self, a: AttentionConfig) -> Dict[str, Any]:
        p: Dict[str, Any] = dict(hidden_size=self.width, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim,
                                 value_dim=a.vdim, scale=a.scale, position=None, names=dict(q="q", k="k", v="v", o="o"))
        if a.chunk is not None:
            p.update(chunk=a.chunk, bias=True, output_gate=True)
            p["names"]["gate"] = "g"
            if a.rot_dims:
                p["position"] = dict(kind="rope_neox", theta=a.rot_base, rotary_dim=a.rot_dims)
                if a.rot_scaling is not None:
                    p["position"].update(kind="rope_banded", **dict(zip(SCALING_KEYS, a.rot_scaling)))
            return p
        p.update(qk_norm="unit", qk_norm_eps=self.norm_eps, taps=a.conv,
                 query_temperature=None if a.q_temp is None else dict(zip(("coef", "every"), a.q_temp)))
        return p

    def _mixer(self, l: NiresunLayer, p: str) -> PartSpec:
        W, eps, m = self.width, self.norm_eps, l.mixer
        if l.type == "mamba1":
            return PartSpec(kind="mamba1", prefix=p, params=dict(
                hidden_size=W, inner=m.inner, state_dim=m.state, dt_rank=m.dt_rank, taps=m.conv))
        if l.type == "attention":
            return PartSpec(kind="attention", prefix=p, params=self._attention(m))
        memory = dict(hidden_size=W, num_heads=m.right.heads, head_dim=m.right.dim, value_dim=m.right.vdim,
                      gate_cap=m.right.gate_cap, eps=eps)
        return PartSpec(kind="side_by_side", prefix=p, params=dict(members=[
            dict(kind="attention", params=self._attention(m.left), prefix="left.", weight=0.5,
                 out_norm=dict(tensor="out", size=W, eps=eps)),
            dict(kind="mlstm", params=memory, prefix="right.", weight=0.5, out_norm=dict(tensor="out", size=W, eps=eps))]))

    def to_spec(self) -> ModelSpec:
        W = self.width
        blocks: List[BlockSpec] = []

        def norm(prefix: str, name: str) -> PartSpec:
            return PartSpec(kind="dynamic_tanh", prefix=prefix, params=dict(size=W, tensor=name))

        for i, l in enumerate(self.layers):
            p = f"l{i}."
            parts: Dict[str, PartSpec] = {"mixer": self._mixer(l, p + "mix."), "mixer_norm": norm(p, "norm1")}
            if l.ff:
                parts.update(feed_forward=PartSpec(kind="swiglu", prefix=p + "mlp.", params=dict(
                    hidden_size=W, intermediate_size=l.ff, activation="gelu_tanh",
                    names=dict(gate="gate", up="up", down="down"))), feed_forward_norm=norm(p, "norm2"))
            blocks.append(BlockSpec("pre_norm", parts))
        spec = ModelSpec(
            architecture="Niresun", vocab_size=self.vocab, hidden_size=W, max_positions=MAX_POSITIONS,
            blocks=tuple(blocks), schedule=default_schedule(len(blocks)),
            embedding=PartSpec(kind="embedding", prefix="", params=dict(vocab_size=self.vocab, hidden_size=W, tensor="embed")),
            final_norm=norm("final.", "norm"),
            head=PartSpec(kind="linear_head", prefix="", params=dict(vocab_size=self.vocab, hidden_size=W, tensor="head")),
            stop_token_ids=self.eos_token_ids,
        )
        spec.validate()
        return spec

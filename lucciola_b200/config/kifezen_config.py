"""Typed configuration of the Kifezen decoder, read from config.json.

Kifezen is a pre-norm decoder on several residual streams (hyper-connections): every sublayer has learned numbers that say
how it reads the streams and how they are mixed and written behind it.  The norms store their weights around zero.  A
layer's mixer is softmax attention on unit queries and keys without rotation, whose queries have a temperature that grows
with their position, or latent attention with a rotated part, a learned sink a head and YaRN-scaled frequencies; both gate
every head with one sigmoid.  A feed-forward is gated (silu), or routed experts weighted by the softmax over the chosen.

    architecture   "Kifezen"
    vocab, width, streams
    norm           {eps}
    layers         [{type, mixer: {...}, mlp: {...} | null}, ...]
        attention mixer:         heads, kv_heads, dim, vdim, scale, q_temp: {coef, every}     (q_temp may be null or absent)
        latent_attention mixer:  heads, dim, rot_dim, vdim, kv_rank, scale, rot: {dims, base, scaling: {factor, original, fast, slow}}
                                 (rot and rot.scaling may be null or absent)
        mlp:  {kind: "dense", ff}, or {kind: "moe", router: {experts, top}, expert: {ff}}

Every size and constant comes from the file; an unknown layer type or feed-forward kind is refused.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from .model_config import ConfigError, _as_float, _as_int
from .riruzen_config import _need, _section
from .venitar_config import RotarySpec, _rotary

ATTENTION = "attention"
LATENT_ATTENTION = "latent_attention"
DENSE = "dense"
MOE = "moe"


@dataclass(frozen=True)
class UnitAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 0             # 0: queries have no temperature


@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int                        # unrotated query/key entries of a head
    rot_dim: int                    # rotated entries, whose key part all heads share
    vdim: int
    kv_rank: int
    scale: float
    rot: RotarySpec = RotarySpec()


@dataclass(frozen=True)
class GatedFeedForwardSpec:
    kind: str                       # "dense" | "moe"
    ff: int                         # the dense layer's, or an expert's
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class KifezenLayer:
    type: str
    attention: Optional[UnitAttentionSpec] = None
    latent: Optional[LatentAttentionSpec] = None
    mlp: Optional[GatedFeedForwardSpec] = None


def _unit_attention(m: Mapping[str, Any], where: str) -> UnitAttentionSpec:
    _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    coef, every = 0.0, 0
    if m.get("q_temp") is not None:
        t = _section(m, "q_temp", where)
        _need(t, ("coef", "every"), f"{where}.q_temp")
        coef, every = _as_float(t, "coef"), _as_int(t, "every")
        if every <= 0:
            raise ConfigError(f"{where}.q_temp: every must be positive, got {every}")
    return UnitAttentionSpec(_as_int(m, "heads"), _as_int(m, "kv_heads"), _as_int(m, "dim"), _as_int(m, "vdim"), _as_float(m, "scale"), coef, every)


def _latent_attention(m: Mapping[str, Any], where: str) -> LatentAttentionSpec:
    _need(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"), where)
    return LatentAttentionSpec(_as_int(m, "heads"), _as_int(m, "dim"), _as_int(m, "rot_dim"), _as_int(m, "vdim"), _as_int(m, "kv_rank"),
                               _as_float(m, "scale"), _rotary(m, where))


def _feed_forward(f: Mapping[str, Any], where: str) -> GatedFeedForwardSpec:
    _need(f, ("kind",), where)
    if f["kind"] == DENSE:
        _need(f, ("ff",), where)
        return GatedFeedForwardSpec(DENSE, _as_int(f, "ff"))
    if f["kind"] != MOE:
        raise ConfigError(f"{where}: unknown kind {f['kind']!r}; known: {DENSE}, {MOE}")
    _need(f, ("router", "expert"), where)
    router, expert = _section(f, "router", where), _section(f, "expert", where)
    _need(router, ("experts", "top"), f"{where}.router")
    _need(expert, ("ff",), f"{where}.expert")
    return GatedFeedForwardSpec(MOE, _as_int(expert, "ff"), _as_int(router, "experts"), _as_int(router, "top"))


@dataclass(frozen=True)
class KifezenConfig:
    architecture: str
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: tuple[KifezenLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Kifezen"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "KifezenConfig":
        _need(d, ("vocab", "width", "streams", "norm", "layers"), "config.json")
        norm = _section(d, "norm")
        _need(norm, ("eps",), "config.json: norm")
        if not isinstance(d["layers"], (list, tuple)) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a list with one entry a layer")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"config.json: layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where} must be an object")
            _need(entry, ("type", "mixer"), where)
            kind, m = entry["type"], _section(entry, "mixer", where)
            mlp = _feed_forward(_section(entry, "mlp", where), f"{where}.mlp") if entry.get("mlp") is not None else None
            if kind == ATTENTION:
                layers.append(KifezenLayer(kind, attention=_unit_attention(m, f"{where}.mixer"), mlp=mlp))
            elif kind == LATENT_ATTENTION:
                layers.append(KifezenLayer(kind, latent=_latent_attention(m, f"{where}.mixer"), mlp=mlp))
            else:
                raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {ATTENTION}, {LATENT_ATTENTION}")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (tuple(int(x) for x in eos) if isinstance(eos, (list, tuple)) else (int(eos),))
        cfg = cls(architecture=cls.ARCHITECTURE, vocab=_as_int(d, "vocab"), width=_as_int(d, "width"), streams=_as_int(d, "streams"),
                  norm_eps=_as_float(norm, "eps"), layers=tuple(layers), eos_token_ids=eos_ids, raw=dict(d))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.streams <= 0:
            raise ConfigError(f"vocab, width and streams must be positive, got {self.vocab}, {self.width}, {self.streams}")
        if not (self.norm_eps > 0):
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        for i, l in enumerate(self.layers):
            where = f"layers[{i}]"
            if l.attention is not None:
                a = l.attention
                if min(a.heads, a.kv_heads, a.dim, a.vdim) <= 0:
                    raise ConfigError(f"{where}: sizes must be positive, got {a}")
                if a.heads % a.kv_heads:
                    raise ConfigError(f"{where}: {a.heads} query heads are not a multiple of {a.kv_heads} kv heads")
            else:
                a = l.latent
                if min(a.heads, a.dim, a.vdim, a.kv_rank) <= 0 or a.rot_dim < 0:
                    raise ConfigError(f"{where}: sizes must be positive, got {a}")
                r = a.rot
                if r.dims < 0 or r.dims % 2 or r.dims > a.rot_dim:
                    raise ConfigError(f"{where}: rot.dims {r.dims} must be even and at most rot_dim {a.rot_dim}")
                if r.dims and not (r.base > 0):
                    raise ConfigError(f"{where}: rot.base must be positive, got {r.base}")
                if r.factor and not (r.factor > 0 and r.original > 0 and r.fast > 0 and r.slow > 0 and r.base != 1):
                    raise ConfigError(f"{where}: rot.scaling wants positive factor, original, fast and slow, and a base other than 1")
            f = l.mlp
            if f is not None and (f.ff <= 0 or (f.kind == MOE and not 0 < f.top <= f.experts)):
                raise ConfigError(f"{where}.mlp: sizes must be positive and top at most experts, got {f}")

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            if l.attention is not None:
                a = l.attention
                m: dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.temp_every:
                    m["q_temp"] = {"coef": a.temp_coef, "every": a.temp_every}
            else:
                b = l.latent
                m = {"heads": b.heads, "dim": b.dim, "rot_dim": b.rot_dim, "vdim": b.vdim, "kv_rank": b.kv_rank, "scale": b.scale}
                if b.rot.dims:
                    m["rot"] = {"dims": b.rot.dims, "base": b.rot.base}
                    if b.rot.factor:
                        m["rot"]["scaling"] = {"factor": b.rot.factor, "original": b.rot.original, "fast": b.rot.fast, "slow": b.rot.slow}
            f = l.mlp
            mlp: Optional[dict[str, Any]] = None
            if f is not None:
                mlp = {"kind": DENSE, "ff": f.ff} if f.kind == DENSE else {"kind": MOE, "router": {"experts": f.experts, "top": f.top},
                                                                            "expert": {"ff": f.ff}}
            layers.append({"type": l.type, "mixer": m, "mlp": mlp})
        d: dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                             "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

"""Typed configuration of the Nulalorn decoder, read from config.json.

Nulalorn is a decoder with a norm in front of and a norm behind every sublayer, x += n1b(mixer(n1(x))); x += n2b(ff(n2(x)))
(a layer may have no feed-forward), of which a run of layers may be repeated: layers loop.start .. loop.stop - 1 run
loop.times times in a row with the same weights and a cache of their own for every pass, and in front of every pass the
stream is mixed with the embedding's output by one linear map and a vector of the pass is added.  Every mixer is softmax
attention over a sliding window whose queries and keys are rotated in pairs of neighbours and then divided by their root
mean square, with a capped score.  A feed-forward is dense, down(gelu(up h)), or a set of such experts named by a table of
the token ids (no router), with one that every token uses behind a sigmoid gate.  The logits are capped.

    architecture   "Nulalorn"
    vocab, width
    norm           {eps}
    logit_softcap                                                (null or absent: the logits are not capped)
    loop           {start, stop, times}                          (null or absent: no loop)
    layers         [{type: "attention", mixer: {...}, mlp: {...} | null}, ...]
        mixer:  heads, kv_heads, dim, vdim, scale, softcap, mask: {size}, rot: {dims, base, scaling: {factor, low, high, original}}
                (softcap, mask, rot and rot.scaling may be null or absent)
        mlp:    {kind: "dense", ff}, or
                {kind: "moe", router: {experts, top}, expert: {ff}, shared: {ff} | null}

Every size and constant comes from the file; an unknown layer type or feed-forward kind is refused.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from .model_config import ConfigError, _as_float, _as_int
from .riruzen_config import _need, _section

ATTENTION = "attention"
DENSE = "dense"
MOE = "moe"


@dataclass(frozen=True)
class NeighbourRotarySpec:
    dims: int = 0                   # 0: no rotation
    base: float = 10000.0
    factor: float = 0.0             # > 0: frequencies scaled by wavelength with the three numbers below
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0


@dataclass(frozen=True)
class CappedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float                  # 0: scores are not capped
    window: int                     # mask.size; 0: plain causal
    rot: NeighbourRotarySpec


@dataclass(frozen=True)
class FeedForwardSpec:
    kind: str                       # "dense" | "moe"
    ff: int                         # the dense layer's, or an expert's
    experts: int = 0
    top: int = 0
    shared_ff: int = 0              # 0: no expert that every token uses


@dataclass(frozen=True)
class NulalornLayer:
    type: str
    attention: CappedAttentionSpec
    mlp: Optional[FeedForwardSpec] = None


def _rotary(m: Mapping[str, Any], where: str) -> NeighbourRotarySpec:
    if m.get("rot") is None:
        return NeighbourRotarySpec()
    rot = _section(m, "rot", where)
    _need(rot, ("dims", "base"), f"{where}.rot")
    if rot.get("scaling") is None:
        return NeighbourRotarySpec(_as_int(rot, "dims"), _as_float(rot, "base"))
    sc = _section(rot, "scaling", f"{where}.rot")
    _need(sc, ("factor", "low", "high", "original"), f"{where}.rot.scaling")
    return NeighbourRotarySpec(_as_int(rot, "dims"), _as_float(rot, "base"), _as_float(sc, "factor"), _as_float(sc, "low"),
                               _as_float(sc, "high"), _as_float(sc, "original"))


def _attention(m: Mapping[str, Any], where: str) -> CappedAttentionSpec:
    _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    window = 0
    if m.get("mask") is not None:
        mask = _section(m, "mask", where)
        _need(mask, ("size",), f"{where}.mask")
        window = _as_int(mask, "size")
    cap = _as_float(m, "softcap") if m.get("softcap") is not None else 0.0
    return CappedAttentionSpec(_as_int(m, "heads"), _as_int(m, "kv_heads"), _as_int(m, "dim"), _as_int(m, "vdim"), _as_float(m, "scale"),
                               cap, window, _rotary(m, where))


def _feed_forward(f: Mapping[str, Any], where: str) -> FeedForwardSpec:
    _need(f, ("kind",), where)
    if f["kind"] == DENSE:
        _need(f, ("ff",), where)
        return FeedForwardSpec(DENSE, _as_int(f, "ff"))
    if f["kind"] != MOE:
        raise ConfigError(f"{where}: unknown kind {f['kind']!r}; known: {DENSE}, {MOE}")
    _need(f, ("router", "expert"), where)
    router, expert = _section(f, "router", where), _section(f, "expert", where)
    _need(router, ("experts", "top"), f"{where}.router")
    _need(expert, ("ff",), f"{where}.expert")
    shared = 0
    if f.get("shared") is not None:
        s = _section(f, "shared", where)
        _need(s, ("ff",), f"{where}.shared")
        shared = _as_int(s, "ff")
        if shared <= 0:
            raise ConfigError(f"{where}.shared: ff must be positive, got {shared}")
    return FeedForwardSpec(MOE, _as_int(expert, "ff"), _as_int(router, "experts"), _as_int(router, "top"), shared)


@dataclass(frozen=True)
class NulalornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[NulalornLayer, ...]
    logit_softcap: float = 0.0      # 0: the logits are not capped
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    eos_token_ids: tuple[int, ...] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False)

    ARCHITECTURE = "Nulalorn"

    @property
    def loops(self) -> bool:
        """Whether a run of layers is looped (a loop of one pass counts: its entry is still in front of it)."""
        return self.loop_stop > self.loop_start

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "NulalornConfig":
        _need(d, ("vocab", "width", "norm", "layers"), "config.json")
        norm = _section(d, "norm")
        _need(norm, ("eps",), "config.json: norm")
        start, stop, times = 0, 0, 1
        if d.get("loop") is not None:
            loop = _section(d, "loop")
            _need(loop, ("start", "stop", "times"), "config.json: loop")
            start, stop, times = _as_int(loop, "start"), _as_int(loop, "stop"), _as_int(loop, "times")
        if not isinstance(d["layers"], (list, tuple)) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a list with one entry a layer")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"config.json: layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where} must be an object")
            _need(entry, ("type", "mixer"), where)
            if entry["type"] != ATTENTION:
                raise ConfigError(f"{where}: unknown layer type {entry['type']!r}; known: {ATTENTION}")
            mlp = _feed_forward(_section(entry, "mlp", where), f"{where}.mlp") if entry.get("mlp") is not None else None
            layers.append(NulalornLayer(ATTENTION, _attention(_section(entry, "mixer", where), f"{where}.mixer"), mlp))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (tuple(int(x) for x in eos) if isinstance(eos, (list, tuple)) else (int(eos),))
        cfg = cls(architecture=cls.ARCHITECTURE, vocab=_as_int(d, "vocab"), width=_as_int(d, "width"), norm_eps=_as_float(norm, "eps"),
                  layers=tuple(layers), logit_softcap=_as_float(d, "logit_softcap") if d.get("logit_softcap") is not None else 0.0,
                  loop_start=start, loop_stop=stop, loop_times=times, eos_token_ids=eos_ids, raw=dict(d))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError(f"vocab and width must be positive, got {self.vocab}, {self.width}")
        if not (self.norm_eps > 0):
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps}")
        if self.logit_softcap < 0:
            raise ConfigError(f"logit_softcap must be positive, got {self.logit_softcap}")
        if not (0 <= self.loop_start <= self.loop_stop <= len(self.layers)) or self.loop_times < 1:
            raise ConfigError(f"loop {self.loop_start}..{self.loop_stop} x {self.loop_times} does not fit {len(self.layers)} layers")
        for i, l in enumerate(self.layers):
            a, where = l.attention, f"layers[{i}]"
            if min(a.heads, a.kv_heads, a.dim, a.vdim) <= 0 or a.window < 0 or a.softcap < 0:
                raise ConfigError(f"{where}: sizes must be positive, window and cap not negative, got {a}")
            if a.heads % a.kv_heads:
                raise ConfigError(f"{where}: {a.heads} query heads are not a multiple of {a.kv_heads} kv heads")
            r = a.rot
            if r.dims < 0 or r.dims % 2 or r.dims > a.dim:
                raise ConfigError(f"{where}: rot.dims {r.dims} must be even and at most dim {a.dim}")
            if r.dims and not (r.base > 0):
                raise ConfigError(f"{where}: rot.base must be positive, got {r.base}")
            if r.factor and not (r.factor > 0 and r.low > 0 and r.high > 0 and r.original > 0):
                raise ConfigError(f"{where}: rot.scaling wants positive factor, low, high and original")
            f = l.mlp
            if f is not None and (f.ff <= 0 or (f.kind == MOE and not 0 < f.top <= f.experts)):
                raise ConfigError(f"{where}.mlp: sizes must be positive and top at most experts, got {f}")

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            a, f = l.attention, l.mlp
            mixer: dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.softcap:
                mixer["softcap"] = a.softcap
            if a.window:
                mixer["mask"] = {"size": a.window}
            if a.rot.dims:
                mixer["rot"] = {"dims": a.rot.dims, "base": a.rot.base}
                if a.rot.factor:
                    mixer["rot"]["scaling"] = {"factor": a.rot.factor, "low": a.rot.low, "high": a.rot.high, "original": a.rot.original}
            mlp: Optional[dict[str, Any]] = None
            if f is not None and f.kind == DENSE:
                mlp = {"kind": DENSE, "ff": f.ff}
            elif f is not None:
                mlp = {"kind": MOE, "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        d: dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                             "layers": layers}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        if self.loops:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

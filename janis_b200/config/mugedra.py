"""Mugedra's configuration: the keys of its config.json, typed.

config.json names the architecture under `architecture` and nests its values:

    vocab, width, norm.eps, loop: {start, stop, times} (optional),
    layers: [ {type: "parallel", mixer: {left: {...}, right: {...}}, mlp: {...} | null}, ... ]

A mixer's `left` is softmax attention: heads, kv_heads, dim (queries and keys), vdim, scale, softcap (0 or absent: none),
mask.size (keys are seen inside chunks of that many positions; absent: everywhere), rot.base, rot.dims and optionally
rot.scaling with factor, original, fast and slow.  `right` is the gated delta rule: heads, kv_heads (heads of queries and
keys), dim, vdim, conv (taps of its short convolutions).  A feed-forward is a mixture of experts ({kind: "moe", expert.ff,
router: {experts, top}}).  Layers start .. stop - 1 of a loop run `times` times in a row.  Every size and constant of a model
comes from here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, ConfigReader
from .larulorn import RampScaling
from .sigalorn import _sub


@dataclass(frozen=True)
class ChunkedHeadsSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float                 # 0: scores are not capped
    chunk: int                     # 0: all earlier keys are seen
    rot_base: float
    rot_dims: int                  # 0: nothing turns
    rot_scaling: RampScaling | None = None

    def to_dict(self) -> dict:
        d: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                d["rot"]["scaling"] = self.rot_scaling.to_dict()
        return d


@dataclass(frozen=True)
class DeltaRuleSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class PairSpec:
    left: ChunkedHeadsSpec
    right: DeltaRuleSpec

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class InputWeightedMoeSpec:
    experts: int
    top: int
    expert_ff: int
    kind: str = "moe"

    def to_dict(self) -> dict:
        return {"kind": self.kind, "expert": {"ff": self.expert_ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class LayerSpec:
    type: str                      # "parallel"
    mixer: Any
    mlp: Any                       # InputWeightedMoeSpec | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int

    def to_dict(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


def _heads_over(r: ConfigReader) -> tuple[int, int]:
    heads = r.integer("heads", minimum=1)
    kv = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv:
        raise ConfigError(f"{r.where}: heads ({heads}) not divisible by kv_heads ({kv})")
    return heads, kv


def _attention(r: ConfigReader) -> ChunkedHeadsSpec:
    heads, kv = _heads_over(r)
    dim = r.integer("dim", minimum=1)
    rot = _sub(r, "rot", required=False)
    base, dims, scaling = 10000.0, 0, None
    if rot is not None:
        base = rot.number("base", default=10000.0, minimum=0.0, exclusive=True)
        dims = rot.integer("dims", default=dim, minimum=0)
        sc = _sub(rot, "scaling", required=False)
        if sc is not None:
            scaling = RampScaling(**{k: sc.number(k, minimum=0.0, exclusive=True) for k in ("factor", "original", "fast", "slow")})
            if base == 1.0:
                raise ConfigError(f"{r.where}: rot.scaling needs a base other than 1")
    if dims % 2 or dims > dim:
        raise ConfigError(f"{r.where}: rot.dims must be even and at most dim ({dim}), found {dims}")
    mask = _sub(r, "mask", required=False)
    return ChunkedHeadsSpec(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                            scale=r.number("scale", default=dim ** -0.5, minimum=0.0, exclusive=True),
                            softcap=r.number("softcap", default=0.0, minimum=0.0),
                            chunk=mask.integer("size", minimum=1) if mask is not None else 0, rot_base=base, rot_dims=dims,
                            rot_scaling=scaling)


def _delta_rule(r: ConfigReader) -> DeltaRuleSpec:
    heads, kv = _heads_over(r)
    dim = r.integer("dim", minimum=1)
    return DeltaRuleSpec(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                         conv=r.integer("conv", minimum=1))


def _parallel(r: ConfigReader) -> PairSpec:
    left, right = _sub(r, "left"), _sub(r, "right")
    left.where, right.where = f"{r.where}.left", f"{r.where}.right"
    return PairSpec(_attention(left), _delta_rule(right))


_MIXERS = {"parallel": _parallel}


def _mlp(fr: ConfigReader) -> InputWeightedMoeSpec:
    kind = fr.string("kind", default="moe")
    if kind != "moe":
        raise ConfigError(f"{fr.where}: unknown kind {kind!r} (known: moe)")
    rr = _sub(fr, "router")
    experts, top = rr.integer("experts", minimum=1), rr.integer("top", minimum=1)
    if top > experts:
        raise ConfigError(f"{fr.where}: top ({top}) exceeds the experts ({experts})")
    return InputWeightedMoeSpec(experts=experts, top=top, expert_ff=_sub(fr, "expert").integer("ff", minimum=1))


@dataclass(frozen=True)
class MugedraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[LayerSpec, ...]
    loop: LoopSpec | None = None
    architecture: str = "Mugedra"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str = "config.json") -> "MugedraConfig":
        r = ConfigReader(raw, where)
        norm = _sub(r, "norm", required=False)
        listed = r.raw.get("layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers: list[LayerSpec] = []
        for i, entry in enumerate(listed):
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where}: layers[{i}] must be an object")
            lr = ConfigReader(entry, f"{where}: layers[{i}]")
            kind = lr.string("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{where}: layers[{i}]: unknown layer type {kind!r} (known: {', '.join(_MIXERS)})")
            mr = _sub(lr, "mixer")
            mr.where = f"{where}: layers[{i}].mixer"
            fr = _sub(lr, "mlp", required=False)
            if fr is not None:
                fr.where = f"{where}: layers[{i}].mlp"
            layers.append(LayerSpec(kind, _MIXERS[kind](mr), _mlp(fr) if fr is not None else None))
        lp = _sub(r, "loop", required=False)
        loop = None
        if lp is not None:
            loop = LoopSpec(start=lp.integer("start", minimum=0), stop=lp.integer("stop", minimum=1), times=lp.integer("times", minimum=1))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"{where}: a loop over layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=norm.number("eps", default=1e-6, minimum=0.0) if norm is not None else 1e-6,
                   layers=tuple(layers), loop=loop, architecture=r.string("architecture", default="Mugedra"))

    def to_dict(self) -> dict:
        """The config.json that reads back to this object."""
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [l.to_dict() for l in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        return d

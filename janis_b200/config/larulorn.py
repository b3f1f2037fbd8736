"""Larulorn's configuration: the keys of its config.json, typed.

config.json names the architecture under `architecture` and nests its values:

    vocab, width, norm.eps, logit_scale,
    layers: [ {type: "attention" | "parallel", mixer: {...}, mlp: {...} | null}, ... ]

An "attention" mixer gives heads, kv_heads, dim (queries and keys), vdim, scale, v_mix (whether the layer's values are
mixed with those of the first layer that says so), rot.base, rot.dims and optionally rot.scaling with factor, original,
fast and slow.  A "parallel" mixer gives two mixers that read the same input, `left`, attention with the same keys (without
v_mix), and `right`, a gated linear recurrence (width, blocks, conv: the taps of its short convolution), and the constants
left_scale and right_scale.  A feed-forward is dense ({kind: "dense", ff, limit}) or a mixture of experts ({kind: "moe",
expert.ff, router: {experts, top, groups: {count, keep} | null}, shared.ff | null}).  Every size and constant of a model
comes from here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, ConfigReader
from .sigalorn import _sub


@dataclass(frozen=True)
class RampScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class HeadsSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int                  # 0: nothing turns
    rot_scaling: RampScaling | None = None
    v_mix: bool = False

    def to_dict(self) -> dict:
        d: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                d["rot"]["scaling"] = self.rot_scaling.to_dict()
        if self.v_mix:
            d["v_mix"] = True
        return d


@dataclass(frozen=True)
class GatedRecurrenceSpec:
    width: int
    blocks: int
    conv: int

    def to_dict(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class SumSpec:
    left: HeadsSpec
    right: GatedRecurrenceSpec
    left_scale: float
    right_scale: float

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}


@dataclass(frozen=True)
class ClampedDenseSpec:
    ff: int
    limit: float
    kind: str = "dense"

    def to_dict(self) -> dict:
        return {"kind": self.kind, "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class PlainMoeSpec:
    experts: int
    top: int
    group_count: int
    group_keep: int
    expert_ff: int
    shared_ff: int                 # 0: no shared expert
    kind: str = "moe"

    def to_dict(self) -> dict:
        return {"kind": self.kind, "expert": {"ff": self.expert_ff},
                "router": {"experts": self.experts, "top": self.top,
                           "groups": {"count": self.group_count, "keep": self.group_keep}},
                "shared": {"ff": self.shared_ff} if self.shared_ff else None}


@dataclass(frozen=True)
class LayerSpec:
    type: str                      # "attention" | "parallel"
    mixer: Any
    mlp: Any                       # ClampedDenseSpec | PlainMoeSpec | None

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


def _heads(r: ConfigReader) -> HeadsSpec:
    heads = r.integer("heads", minimum=1)
    kv = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv:
        raise ConfigError(f"{r.where}: heads ({heads}) not divisible by kv_heads ({kv})")
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
    return HeadsSpec(heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                     scale=r.number("scale", default=dim ** -0.5, minimum=0.0, exclusive=True), rot_base=base, rot_dims=dims,
                     rot_scaling=scaling, v_mix=r.boolean("v_mix", default=False))


def _recurrence(r: ConfigReader) -> GatedRecurrenceSpec:
    width, blocks = r.integer("width", minimum=1), r.integer("blocks", default=1, minimum=1)
    if width % blocks:
        raise ConfigError(f"{r.where}: width ({width}) not divisible by blocks ({blocks})")
    return GatedRecurrenceSpec(width=width, blocks=blocks, conv=r.integer("conv", minimum=1))


def _parallel(r: ConfigReader) -> SumSpec:
    left, right = _sub(r, "left"), _sub(r, "right")
    left.where, right.where = f"{r.where}.left", f"{r.where}.right"
    heads = _heads(left)
    if heads.v_mix:
        raise ConfigError(f"{left.where}: v_mix belongs to layers of type attention")
    return SumSpec(heads, _recurrence(right), r.number("left_scale", default=1.0), r.number("right_scale", default=1.0))


_MIXERS = {"attention": _heads, "parallel": _parallel}


def _mlp(fr: ConfigReader):
    kind = fr.string("kind", default="dense")
    if kind == "dense":
        return ClampedDenseSpec(ff=fr.integer("ff", minimum=1), limit=fr.number("limit", minimum=0.0, exclusive=True))
    if kind != "moe":
        raise ConfigError(f"{fr.where}: unknown kind {kind!r} (known: dense, moe)")
    rr = _sub(fr, "router")
    experts, top = rr.integer("experts", minimum=1), rr.integer("top", minimum=1)
    gr = _sub(rr, "groups", required=False)
    count = gr.integer("count", default=1, minimum=1) if gr is not None else 1
    keep = gr.integer("keep", default=count, minimum=1) if gr is not None else 1
    if experts % count or keep > count:
        raise ConfigError(f"{fr.where}: {experts} experts in {count} groups of which {keep} are kept")
    if top > keep * (experts // count):
        raise ConfigError(f"{fr.where}: top ({top}) exceeds the experts of the kept groups ({keep * (experts // count)})")
    sh = _sub(fr, "shared", required=False)
    return PlainMoeSpec(experts=experts, top=top, group_count=count, group_keep=keep,
                        expert_ff=_sub(fr, "expert").integer("ff", minimum=1),
                        shared_ff=sh.integer("ff", minimum=1) if sh is not None else 0)


@dataclass(frozen=True)
class LarulornConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: tuple[LayerSpec, ...]
    architecture: str = "Larulorn"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str = "config.json") -> "LarulornConfig":
        r = ConfigReader(raw, where)
        norm = _sub(r, "norm", required=False)
        listed = r.raw.get("layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers: list[LayerSpec] = []
        values = None                            # key/value heads x value size of the layers whose values are mixed
        for i, entry in enumerate(listed):
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where}: layers[{i}] must be an object")
            lr = ConfigReader(entry, f"{where}: layers[{i}]")
            kind = lr.string("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{where}: layers[{i}]: unknown layer type {kind!r} (known: {', '.join(_MIXERS)})")
            mr = _sub(lr, "mixer")
            mr.where = f"{where}: layers[{i}].mixer"
            mixer = _MIXERS[kind](mr)
            if kind == "attention" and mixer.v_mix:
                if values is not None and values != (mixer.kv_heads, mixer.vdim):
                    raise ConfigError(f"{mr.where}: mixed values must have the same heads and size in every layer, "
                                      f"found {mixer.kv_heads} x {mixer.vdim} after {values[0]} x {values[1]}")
                values = (mixer.kv_heads, mixer.vdim)
            fr = _sub(lr, "mlp", required=False)
            if fr is not None:
                fr.where = f"{where}: layers[{i}].mlp"
            layers.append(LayerSpec(kind, mixer, _mlp(fr) if fr is not None else None))
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=norm.number("eps", default=1e-6, minimum=0.0) if norm is not None else 1e-6,
                   logit_scale=r.number("logit_scale", default=1.0), layers=tuple(layers),
                   architecture=r.string("architecture", default="Larulorn"))

    def to_dict(self) -> dict:
        """The config.json that reads back to this object."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "layers": [l.to_dict() for l in self.layers]}

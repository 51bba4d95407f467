"""`GakupelConfig`: the config.json of the Gakupel decoder, typed and checked.

A Gakupel model is a list of layers with the norm on each sublayer's result, x <- x + norm(sublayer(x)), whose results are
averaged over the depth with learned weights:

    architecture    "Gakupel"
    vocab, width
    norm.eps                        of every norm of the model
    max_positions                   optional: the longest sequence (absent: DEFAULT_MAX_POSITIONS)
    layers[i].type                  "attention", "delta" or "parallel"
    layers[i].mixer                 attention: heads, kv_heads, dim, vdim (= dim: the values are the keys), scale,
                                               rot {base, dims} (absent: no rotation)
                                    delta: heads, kv_heads, dim, vdim, conv (taps)
                                    parallel: left {heads, kv_heads, dim, vdim, scale, q_temp {coef, every} (absent: none)},
                                              right {heads, dim, vdim, gate_cap}, left_scale, right_scale (absent: 1)
    layers[i].mlp                   null, {kind: "dense", ff}, or {kind: "moe", expert {ff}, router {experts, top,
                                    groups {count, keep} (absent: none), scale (absent: 1)}, shared {ff} (absent: none)}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, take
from .vegodra import DEFAULT_MAX_POSITIONS, RotaryConfig, _sub


def _optional(d, key, where) -> Optional[dict]:
    v = d.get(key)
    if v is not None and not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key} must be an object or null")
    return v


@dataclass(frozen=True)
class SharedKeyAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryConfig

    @classmethod
    def read(cls, m, where):
        pos = lambda key: take(m, key, int, positive=True)
        dim = pos("dim")
        r = _optional(m, "rot", where)
        rot = RotaryConfig(take(r, "base", float, positive=True), take(r, "dims", int)) if r else RotaryConfig(10000.0, 0)
        if rot.dims < 0 or rot.dims % 2 or rot.dims > dim:
            raise ConfigError(f"config.json: {where}rot.dims = {rot.dims} must be even and at most dim = {dim}")
        c = cls(pos("heads"), pos("kv_heads"), dim, take(m, "vdim", int, dim, positive=True), take(m, "scale", float), rot)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}{c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        if c.vdim != c.dim:
            raise ConfigError(f"config.json: {where}vdim = {c.vdim} must be dim = {c.dim} (the values are the keys)")
        return c

    def to_dict(self):
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.rot.dims:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class GatedDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def read(cls, m, where):
        pos = lambda key: take(m, key, int, positive=True)
        c = cls(pos("heads"), pos("kv_heads"), pos("dim"), pos("vdim"), pos("conv"))
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}{c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        return c

    def to_dict(self):
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, conv=self.conv)


@dataclass(frozen=True)
class QueryTemperatureConfig:
    coef: float
    every: float

    def to_dict(self):
        return dict(coef=self.coef, every=int(self.every) if float(self.every).is_integer() else self.every)


@dataclass(frozen=True)
class DistanceAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperatureConfig] = None

    @classmethod
    def read(cls, m, where):
        pos = lambda key: take(m, key, int, positive=True)
        t = _optional(m, "q_temp", where)
        temp = QueryTemperatureConfig(take(t, "coef", float), take(t, "every", float, positive=True)) if t else None
        c = cls(pos("heads"), pos("kv_heads"), pos("dim"), pos("vdim"), take(m, "scale", float), temp)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}{c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        return c

    def to_dict(self):
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.q_temp is not None:
            d["q_temp"] = self.q_temp.to_dict()
        return d


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def read(cls, m, where):
        pos = lambda key: take(m, key, int, positive=True)
        c = cls(pos("heads"), pos("dim"), pos("vdim"), take(m, "gate_cap", float, positive=True))
        if take(m, "kv_heads", int, c.heads) != c.heads:
            raise ConfigError(f"config.json: {where}kv_heads must be heads = {c.heads} (every head has its own query and key)")
        return c

    def to_dict(self):
        return dict(heads=self.heads, dim=self.dim, vdim=self.vdim, gate_cap=self.gate_cap)


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: DistanceAttentionConfig
    right: MatrixMemoryConfig
    left_scale: float = 1.0
    right_scale: float = 1.0

    @classmethod
    def read(cls, m, where):
        return cls(DistanceAttentionConfig.read(_sub(m, "left", where), where + "left."),
                   MatrixMemoryConfig.read(_sub(m, "right", where), where + "right."),
                   take(m, "left_scale", float, 1.0), take(m, "right_scale", float, 1.0))

    def to_dict(self):
        return dict(left=self.left.to_dict(), right=self.right.to_dict(), left_scale=self.left_scale, right_scale=self.right_scale)


MIXERS = {"attention": SharedKeyAttentionConfig, "delta": GatedDeltaConfig, "parallel": ParallelMixerConfig}


@dataclass(frozen=True)
class GeluFFConfig:
    ff: int

    def to_dict(self):
        return dict(kind="dense", ff=self.ff)


@dataclass(frozen=True)
class GroupedExpertsConfig:
    ff: int
    experts: int
    top: int
    scale: float = 1.0
    groups: Optional[Tuple[int, int]] = None      # (count, keep)
    shared_ff: Optional[int] = None

    @classmethod
    def read(cls, mlp, where):
        r = _sub(mlp, "router", where)
        g, s = _optional(r, "groups", where + "router."), _optional(mlp, "shared", where)
        c = cls(take(_sub(mlp, "expert", where), "ff", int, positive=True), take(r, "experts", int, positive=True),
                take(r, "top", int, positive=True), take(r, "scale", float, 1.0),
                (take(g, "count", int, positive=True), take(g, "keep", int, positive=True)) if g else None,
                take(s, "ff", int, positive=True) if s else None)
        if c.top > c.experts:
            raise ConfigError(f"config.json: {where}router: top = {c.top} of {c.experts} experts")
        if c.groups:
            n, keep = c.groups
            if c.experts % n or keep > n or keep * (c.experts // n) < c.top:
                raise ConfigError(f"config.json: {where}router: {c.experts} experts in {n} groups of which {keep} stay, {c.top} chosen")
        return c

    def to_dict(self):
        router = dict(experts=self.experts, top=self.top, scale=self.scale)
        if self.groups:
            router["groups"] = dict(count=self.groups[0], keep=self.groups[1])
        d = dict(kind="moe", expert=dict(ff=self.ff), router=router)
        if self.shared_ff:
            d["shared"] = dict(ff=self.shared_ff)
        return d


@dataclass(frozen=True)
class GakupelLayerConfig:
    type: str                         # "attention" | "delta" | "parallel"
    mixer: Any
    mlp: Any = None                   # None | GeluFFConfig | GroupedExpertsConfig

    def to_dict(self):
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=None if self.mlp is None else self.mlp.to_dict())


@dataclass(frozen=True)
class GakupelConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[GakupelLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "GakupelConfig":
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = take(L, "type", str)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not known (known: {sorted(MIXERS)})")
            mixer = MIXERS[kind].read(_sub(L, "mixer", where), where + "mixer.")
            mlp, ff = _optional(L, "mlp", where), None
            if mlp is not None:
                k = take(mlp, "kind", str, "dense")
                if k == "dense":
                    ff = GeluFFConfig(take(mlp, "ff", int, positive=True))
                elif k == "moe":
                    ff = GroupedExpertsConfig.read(mlp, where + "mlp.")
                else:
                    raise ConfigError(f"config.json: {where}mlp.kind {k!r} is not known (known: 'dense', 'moe')")
            layers.append(GakupelLayerConfig(kind, mixer, ff))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos)
        return cls(architecture=d["architectures"][0] if "architectures" in d else d["architecture"],
                   vocab=take(d, "vocab", int, positive=True), width=take(d, "width", int, positive=True),
                   norm_eps=take(_sub(d, "norm", ""), "eps", float, positive=True), layers=tuple(layers),
                   max_positions=take(d, "max_positions", int, DEFAULT_MAX_POSITIONS, positive=True), eos_token_ids=eos_ids)

    def to_dict(self) -> Dict[str, Any]:
        d = dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                 layers=[L.to_dict() for L in self.layers])
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

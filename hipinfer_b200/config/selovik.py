"""`SelovikConfig`: the config.json of the Selovik decoder, typed and checked.

A Selovik model is a list of layers, each with two norms of the same rows, x <- x + (mixer(norm1(x)) + ff(norm2(x))), of which
a run of neighbours may be gone through several times with the same weights:

    architecture    "Selovik"
    vocab, width
    norm.eps                        of every norm of the model
    embedding.scale                 multiplies the token embedding (absent: 1)
    embedding.bigram                {buckets, mul_prev, mul_cur}: the table of token pairs (absent: none)
    logit_scale                     multiplies the logits (absent: 1)
    loop                            {start, stop, times}: layers start .. stop - 1 run `times` times (absent: no loop)
    max_positions                   optional: the longest sequence (absent: DEFAULT_MAX_POSITIONS)
    layers[i].type                  "attention" (differential attention)
    layers[i].mixer                 heads, kv_heads, dim (query/key size of a map), vdim, scale, diff (the constant of the
                                    differential combination), rot {base, dims, scaling {factor, original, fast, slow}}
                                    (scaling absent: none; rot absent: no rotation), mask {size} (absent: every earlier token
                                    is seen)
    layers[i].mlp                   null, {kind: "dense", ff}, or {kind: "moe", expert {ff}, router {experts, top, identity
                                    (absent: 0), groups {count, keep} (absent: none)}, shared {ff} (absent: none)}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, take
from .gakupel import _optional
from .mavinex import ScaledRotaryConfig
from .vegodra import DEFAULT_MAX_POSITIONS, _sub


@dataclass(frozen=True)
class RotaryDiffAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: ScaledRotaryConfig
    window: Optional[int] = None      # mask.size; None: no window

    @classmethod
    def read(cls, m, where):
        pos = lambda key: take(m, key, int, positive=True)
        dim, rot = pos("dim"), ScaledRotaryConfig(10000.0, 0)
        r = _optional(m, "rot", where)
        if r:
            sc = _optional(r, "scaling", where + "rot.")
            rot = ScaledRotaryConfig(take(r, "base", float, positive=True), take(r, "dims", int),
                                     tuple((k, take(sc, k, float, positive=True)) for k in ("factor", "fast", "original", "slow"))
                                     if sc else None)
        if rot.dims < 0 or rot.dims % 2 or rot.dims > dim:
            raise ConfigError(f"config.json: {where}rot.dims = {rot.dims} must be even and at most dim = {dim}")
        mask = _optional(m, "mask", where)
        c = cls(pos("heads"), pos("kv_heads"), dim, pos("vdim"), take(m, "scale", float, positive=True), take(m, "diff", float), rot,
                take(mask, "size", int, None, positive=True) if mask else None)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}{c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
        return c

    def to_dict(self):
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale, diff=self.diff)
        if self.rot.dims:
            d["rot"] = self.rot.to_dict()
        if self.window is not None:
            d["mask"] = dict(size=self.window)
        return d


@dataclass(frozen=True)
class SquaredReluFFConfig:
    ff: int

    def to_dict(self):
        return dict(kind="dense", ff=self.ff)


@dataclass(frozen=True)
class IdentityExpertsConfig:
    ff: int
    experts: int
    top: int
    identity: int = 0
    groups: Optional[Tuple[int, int]] = None      # (count, keep), over experts and identity experts together
    shared_ff: Optional[int] = None

    @classmethod
    def read(cls, mlp, where):
        r = _sub(mlp, "router", where)
        g, s = _optional(r, "groups", where + "router."), _optional(mlp, "shared", where)
        c = cls(take(_sub(mlp, "expert", where), "ff", int, positive=True), take(r, "experts", int, positive=True),
                take(r, "top", int, positive=True), take(r, "identity", int, 0),
                (take(g, "count", int, positive=True), take(g, "keep", int, positive=True)) if g else None,
                take(s, "ff", int, positive=True) if s else None)
        n, (count, keep) = c.experts + c.identity, c.groups or (1, 1)
        if c.identity < 0 or n % count or keep > count or keep * (n // count) < c.top:
            raise ConfigError(f"config.json: {where}router: {c.experts} experts and {c.identity} identity experts in {count} groups of "
                              f"which {keep} stay, {c.top} chosen")
        return c

    def to_dict(self):
        router = dict(experts=self.experts, top=self.top)
        if self.identity:
            router["identity"] = self.identity
        if self.groups:
            router["groups"] = dict(count=self.groups[0], keep=self.groups[1])
        d = dict(kind="moe", expert=dict(ff=self.ff), router=router)
        if self.shared_ff:
            d["shared"] = dict(ff=self.shared_ff)
        return d


@dataclass(frozen=True)
class SelovikLayerConfig:
    type: str                         # "attention"
    mixer: RotaryDiffAttentionConfig
    mlp: Any = None                   # None | SquaredReluFFConfig | IdentityExpertsConfig

    def to_dict(self):
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=None if self.mlp is None else self.mlp.to_dict())


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int

    def to_dict(self):
        return dict(start=self.start, stop=self.stop, times=self.times)


@dataclass(frozen=True)
class SelovikConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[SelovikLayerConfig, ...]
    loop: Optional[LoopConfig] = None
    embedding_scale: float = 1.0
    bigram: Optional[Tuple[int, int, int]] = None      # (buckets, mul_prev, mul_cur)
    logit_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    def run_order(self):
        """[(layer, the pass that starts with it or None)] in the order in which the layers run."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, None) for i in range(n)]
        passes = [(i, t if i == loop.start else None) for t in range(loop.times) for i in range(loop.start, loop.stop)]
        return [(i, None) for i in range(loop.start)] + passes + [(i, None) for i in range(loop.stop, n)]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SelovikConfig":
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = take(L, "type", str)
            if kind != "attention":
                raise ConfigError(f"config.json: {where}type {kind!r} is not known (known: 'attention')")
            mixer = RotaryDiffAttentionConfig.read(_sub(L, "mixer", where), where + "mixer.")
            mlp, ff = _optional(L, "mlp", where), None
            if mlp is not None:
                k = take(mlp, "kind", str, "dense")
                if k == "dense":
                    ff = SquaredReluFFConfig(take(mlp, "ff", int, positive=True))
                elif k == "moe":
                    ff = IdentityExpertsConfig.read(mlp, where + "mlp.")
                else:
                    raise ConfigError(f"config.json: {where}mlp.kind {k!r} is not known (known: 'dense', 'moe')")
            layers.append(SelovikLayerConfig(kind, mixer, ff))
        lp, loop = _optional(d, "loop", ""), None
        if lp is not None:
            loop = LoopConfig(take(lp, "start", int), take(lp, "stop", int), take(lp, "times", int, positive=True))
            if not 0 <= loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop: layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        emb = _optional(d, "embedding", "") or {}
        b, bigram = _optional(emb, "bigram", "embedding."), None
        if b is not None:
            bigram = (take(b, "buckets", int, positive=True), take(b, "mul_prev", int), take(b, "mul_cur", int))
            if min(bigram) < 0:
                raise ConfigError("config.json: embedding.bigram: the multipliers must not be negative")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else (int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos)
        return cls(architecture=d["architectures"][0] if "architectures" in d else d["architecture"],
                   vocab=take(d, "vocab", int, positive=True), width=take(d, "width", int, positive=True),
                   norm_eps=take(_sub(d, "norm", ""), "eps", float, positive=True), layers=tuple(layers), loop=loop,
                   embedding_scale=take(emb, "scale", float, 1.0), bigram=bigram, logit_scale=take(d, "logit_scale", float, 1.0),
                   max_positions=take(d, "max_positions", int, DEFAULT_MAX_POSITIONS, positive=True), eos_token_ids=eos_ids)

    def to_dict(self) -> Dict[str, Any]:
        d = dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                 embedding=dict(scale=self.embedding_scale), logit_scale=self.logit_scale, layers=[L.to_dict() for L in self.layers])
        if self.bigram is not None:
            d["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

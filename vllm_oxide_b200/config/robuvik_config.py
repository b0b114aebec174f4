"""Typed configuration of the Robuvik decoder, read from config.json's own keys.

A Robuvik model is a list of layers in which the mixer and the feed-forward read one norm side by side. A layer's mixer is
`attention` (grouped heads, biases on q, k and v, partial rotary positions, a sliding window, a softmax with one more in its
denominator) or `latent_attention` (a cached latent vector per token with a shared rotated key part, queries through a latent
of their own, an output gate); both stretch their rotary positions where `rot.scaling` is given. The feed-forward is dense
(relu squared), a mixture of small gated experts that read their weight times the input, beside a shared expert, or absent. A
vector per pair of neighbouring tokens is added to the embedding. A range of the layers (`loop`) runs several times with the
same weights and caches of its own each time; every pass begins with a learned vector, and every pass but the first with the
embedding's output once more.

    {"architecture": "Robuvik", "vocab": ..., "width": ..., "norm": {"eps": ...},
     "embedding": {"bigram": {"buckets": ..., "mul_prev": ..., "mul_cur": ...}},
     "loop": {"start": ..., "stop": ..., "times": ...},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                           "rot": {"dims", "base", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": {"kind": "dense", "ff": ...}},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {...}},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"}}}]}

Every size and every constant that may differ between two models of the design is read here. Optional keys: `embedding` and
`bigram` (absent: the token's row alone), `loop` (absent: every layer runs once), `mask` (absent: every earlier token is seen),
`rot` of an attention layer (absent: no rotation), `rot.scaling` (absent: plain frequencies), `shared`, `mlp` (null: no
feed-forward).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..errors import ConfigError
from .lomopel_config import _heads
from .model_config import _need, _typed
from .pironex_config import _positive
from .rotepel_config import _obj

NAME = "Robuvik"
LAYER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class StretchedRotaryConfig:
    """Rotary positions on `dims` features of a head; with `factor` the frequencies are stretched."""
    dims: int
    base: float
    factor: Optional[float] = None        # None: plain frequencies
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    @classmethod
    def from_dict(cls, r: dict, where: str, dims: Optional[int] = None) -> "StretchedRotaryConfig":
        """`dims`: the number of features that are rotated where the mixer fixes it ('dims' may then be left out)."""
        n = dims if dims is not None and r.get("dims") is None else _need(r, "dims", int, where)
        if dims is not None and n != dims:
            raise ConfigError(f"{where}: 'dims' must equal 'rot_dim' ({dims})")
        kw = dict(dims=n, base=_need(r, "base", float, where))
        sc = _obj(r, "scaling", where, optional=True)
        if sc is not None:
            w = where + ".scaling"
            kw.update({k: _need(sc, k, float, w) for k in ("factor", "original", "fast", "slow")})
            _positive(w, factor=kw["factor"], original=kw["original"], fast=kw["fast"], slow=kw["slow"])
        if n < 0 or n % 2 or kw["base"] <= 0 or (sc is not None and kw["base"] == 1):
            raise ConfigError(f"{where}: {n} rotated features (an even number) with base {kw['base']} (positive, not 1 where stretched)")
        return cls(**kw)

    def to_dict(self) -> dict:
        d = {"dims": self.dims, "base": self.base}
        if self.factor is not None:
            d["scaling"] = {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}
        return d


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[StretchedRotaryConfig] = None
    window: int = 0                       # tokens a query sees, itself included; 0: all earlier ones

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "WindowAttentionConfig":
        kw = _heads(m, where)
        kw["scale"] = _need(m, "scale", float, where)
        rot = _obj(m, "rot", where, optional=True)
        if rot is not None:
            kw["rot"] = StretchedRotaryConfig.from_dict(rot, where + ".rot")
            if kw["rot"].dims > kw["dim"]:
                raise ConfigError(f"{where}.rot: {kw['rot'].dims} rotated features of a head of {kw['dim']}")
        mask = _obj(m, "mask", where, optional=True)
        if mask is not None:
            kw["window"] = _need(mask, "size", int, where + ".mask")
            _positive(where + ".mask", size=kw["window"])
        return cls(**kw)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class GatedLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: StretchedRotaryConfig

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "GatedLatentConfig":
        kw = {k: _need(m, k, int, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
        _positive(where, **kw)
        kw["scale"] = _need(m, "scale", float, where)
        kw["rot"] = StretchedRotaryConfig.from_dict(_obj(m, "rot", where), where + ".rot", dims=kw["rot_dim"])
        return cls(**kw)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
                "q_rank": self.q_rank, "scale": self.scale, "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class DenseOrExpertsConfig:
    kind: str                             # "dense" or "moe"
    ff: int                               # hidden size of the dense layer, or of one expert
    experts: int = 0
    top: int = 0
    shared_ff: int = 0                    # 0: no shared expert

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "DenseOrExpertsConfig":
        kind = m.get("kind")
        if kind == "dense":
            c = cls(kind=kind, ff=_need(m, "ff", int, where))
        elif kind == "moe":
            r = _obj(m, "router", where)
            sh = _obj(m, "shared", where, optional=True)
            c = cls(kind=kind, ff=_need(_obj(m, "expert", where), "ff", int, where + ".expert"),
                    experts=_need(r, "experts", int, where + ".router"), top=_need(r, "top", int, where + ".router"),
                    shared_ff=_need(sh, "ff", int, where + ".shared") if sh is not None else 0)
            if not 0 < c.top <= c.experts:
                raise ConfigError(f"{where}.router: {c.top} choices among {c.experts} experts")
            if sh is not None:
                _positive(where + ".shared", ff=c.shared_ff)
        else:
            raise ConfigError(f"{where}: kind {kind!r} is not known (dense or moe)")
        _positive(where, ff=c.ff)
        return c

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        d = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class RobuvikLayer:
    type: str
    attention: Optional[WindowAttentionConfig] = None
    latent: Optional[GatedLatentConfig] = None
    mlp: Optional[DenseOrExpertsConfig] = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "RobuvikLayer":
        if not isinstance(d, dict):
            raise ConfigError(f"{where}: a layer must be an object")
        kind = d.get("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}: 'type' must be one of {', '.join(LAYER_TYPES)}, got {kind!r}")
        m = _obj(d, "mixer", where)
        mlp = _obj(d, "mlp", where, optional=True)
        mixer = dict(attention=WindowAttentionConfig.from_dict(m, where + ".mixer")) if kind == "attention" else \
            dict(latent=GatedLatentConfig.from_dict(m, where + ".mixer"))
        return cls(type=kind, mlp=DenseOrExpertsConfig.from_dict(mlp, where + ".mlp") if mlp is not None else None, **mixer)

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": (self.attention or self.latent).to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


@dataclass(frozen=True)
class BigramConfig:
    """Row (previous * mul_prev + token * mul_cur) mod buckets of a table of buckets + 1 rows, the last one for first tokens."""
    buckets: int
    mul_prev: int
    mul_cur: int

    @classmethod
    def from_dict(cls, b: dict, where: str) -> "BigramConfig":
        c = cls(**{k: _need(b, k, int, where) for k in ("buckets", "mul_prev", "mul_cur")})
        if c.buckets <= 0 or not 0 <= c.mul_prev < 2 ** 31 or not 0 <= c.mul_cur < 2 ** 31:
            raise ConfigError(f"{where}: 'buckets' must be positive and the factors 0 .. 2^31 - 1")
        return c

    def to_dict(self) -> dict:
        return {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}


@dataclass(frozen=True)
class RobuvikConfig:
    vocab: int
    width: int
    layers: Tuple[RobuvikLayer, ...]
    norm_eps: float
    bigram: Optional[BigramConfig] = None
    loop: Optional[Tuple[int, int, int]] = None     # (start, stop, times)
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, d: dict, where: str = "config.json") -> "RobuvikConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        kw = dict(vocab=_need(d, "vocab", int, where), width=_need(d, "width", int, where),
                  layers=tuple(RobuvikLayer.from_dict(x, f"{where}: layers[{i}]") for i, x in enumerate(layers)),
                  norm_eps=_need(_obj(d, "norm", where), "eps", float, where + ".norm"))
        emb = _obj(d, "embedding", where, optional=True)
        pair = _obj(emb, "bigram", where + ".embedding", optional=True) if emb is not None else None
        if pair is not None:
            kw["bigram"] = BigramConfig.from_dict(pair, where + ".embedding.bigram")
        lp = _obj(d, "loop", where, optional=True)
        if lp is not None:
            kw["loop"] = tuple(_need(lp, k, int, where + ".loop") for k in ("start", "stop", "times"))
        cfg = cls(**kw)
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config") -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError(f"{where}: vocab and width must be positive")
        if self.loop is not None:
            a, b, times = self.loop
            if not 0 <= a < b <= len(self.layers) or times < 1:
                raise ConfigError(f"{where}: loop {self.loop} does not fit {len(self.layers)} layers")

    def run_order(self) -> Tuple[Tuple[int, Optional[int]], ...]:
        """(layer, number of the pass of the loop that begins with this run, or None), in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return tuple((i, None) for i in range(n))
        a, b, times = self.loop
        order = [(i, None) for i in range(a)]
        for r in range(times):
            order += [(i, r if i == a else None) for i in range(a, b)]
        return tuple(order + [(i, None) for i in range(b, n)])

    def param_count(self) -> int:
        from ..models.robuvik import robuvik_manifest
        total = 0
        for spec in robuvik_manifest(self).values():
            n = 1
            for x in spec.shape:
                n *= max(int(x), 0)
            total += n
        return total

    def to_dict(self) -> dict:
        d = {"architecture": NAME, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [x.to_dict() for x in self.layers]}
        if self.bigram is not None:
            d["embedding"] = {"bigram": self.bigram.to_dict()}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

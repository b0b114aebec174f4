"""Typed configuration of the Fanopel decoder, read from config.json's own keys.

A Fanopel model is a list of layers of type `attention`: softmax attention whose values are its keys as projected (norms
over the whole q and k projections, capped scores, a bias that grows linearly with the distance, a sliding window beside
which the first tokens of the sequence stay visible, one sigmoid gate per head) and a mixture of small experts without a
gate (relu squared, sigmoid scores with a correction that only the election sees, groups of experts), or no feed-forward.
Layer norms with a weight sit in front of the sub-layers; what a sub-layer returns is multiplied by one constant before
it joins the residual. A learned vector per position is added to the embedding.

    {"architecture": "Fanopel", "vocab": ..., "width": ..., "max_positions": ..., "norm": {"eps": ...}, "residual_mult": ...,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask": {"size", "keep_first"}},
                 "mlp": {"kind": "moe", "expert": {"ff": ...},
                         "router": {"experts": ..., "top": ..., "scale": ..., "groups": {"count": ..., "keep": ...}}}}]}

Every size and every constant that may differ between two models of the design is read here. Optional keys: `mask`
(absent: every earlier token is seen), `mask.keep_first` (absent or 0: none), `softcap` (absent or 0: scores are not
capped), `vdim` (absent: `dim`; the two are one size), `router.scale` (absent: 1), `groups` (absent: every expert stands
for election), `residual_mult` (absent: 1), `mlp` (null: no feed-forward).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..errors import ConfigError
from .lomopel_config import _heads
from .model_config import _need, _typed
from .rotepel_config import _obj

NAME = "Fanopel"


@dataclass(frozen=True)
class KeyValueAttentionConfig:
    """Attention whose values are its keys."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: float = 0.0                  # 0: scores are not capped
    window: int = 0                       # tokens a query sees, itself included; 0: all earlier ones
    keep_first: int = 0                   # first tokens of the sequence that stay visible behind the window

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "KeyValueAttentionConfig":
        kw = _heads(m if "vdim" in m else {**m, "vdim": m.get("dim")}, where)
        vdim = kw.pop("vdim")
        if vdim != kw["dim"]:
            raise ConfigError(f"{where}: the values are the keys, so 'vdim' {vdim} must be 'dim' {kw['dim']}")
        kw["scale"] = _need(m, "scale", float, where)
        if m.get("softcap") is not None:
            kw["softcap"] = _typed(m, "softcap", float, where)
            if kw["softcap"] < 0:
                raise ConfigError(f"{where}: 'softcap' must not be negative")
        mask = _obj(m, "mask", where, optional=True)
        if mask is not None:
            kw["window"] = _need(mask, "size", int, where + ".mask")
            if kw["window"] <= 0:
                raise ConfigError(f"{where}.mask: 'size' must be positive")
            if mask.get("keep_first") is not None:
                kw["keep_first"] = _typed(mask, "keep_first", int, where + ".mask")
                if kw["keep_first"] < 0:
                    raise ConfigError(f"{where}.mask: 'keep_first' must not be negative")
        return cls(**kw)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim, "scale": self.scale}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.window:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return d


@dataclass(frozen=True)
class PlainExpertsConfig:
    """Routed experts without a gate, elected by sigmoid scores and a correction."""
    ff: int
    experts: int
    top: int
    scale: float = 1.0
    groups: int = 0                       # 0: no groups
    keep: int = 0

    @classmethod
    def from_dict(cls, m: dict, where: str) -> "PlainExpertsConfig":
        if m.get("kind") != "moe":
            raise ConfigError(f"{where}: kind {m.get('kind')!r} is not known (moe)")
        r = _obj(m, "router", where)
        kw = dict(ff=_need(_obj(m, "expert", where), "ff", int, where + ".expert"), experts=_need(r, "experts", int, where + ".router"),
                  top=_need(r, "top", int, where + ".router"))
        if r.get("scale") is not None:
            kw["scale"] = _typed(r, "scale", float, where + ".router")
        g = _obj(r, "groups", where + ".router", optional=True)
        if g is not None:
            kw["groups"] = _need(g, "count", int, where + ".router.groups")
            kw["keep"] = _need(g, "keep", int, where + ".router.groups")
        cfg = cls(**kw)
        if cfg.ff <= 0 or not 0 < cfg.top <= cfg.experts:
            raise ConfigError(f"{where}: experts of {cfg.ff}, {cfg.top} choices among {cfg.experts}")
        if g is not None and (cfg.groups <= 0 or cfg.experts % cfg.groups or not 0 < cfg.keep <= cfg.groups
                              or cfg.top > cfg.keep * (cfg.experts // cfg.groups)):
            raise ConfigError(f"{where}.router: {cfg.experts} experts in {cfg.groups} groups of which {cfg.keep} are kept "
                              f"cannot give {cfg.top} choices")
        return cfg

    def to_dict(self) -> dict:
        r = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.groups:
            r["groups"] = {"count": self.groups, "keep": self.keep}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": r}


@dataclass(frozen=True)
class FanopelLayer:
    attention: KeyValueAttentionConfig
    mlp: Optional[PlainExpertsConfig] = None      # None: the layer has no feed-forward

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "FanopelLayer":
        if not isinstance(d, dict):
            raise ConfigError(f"{where}: a layer must be an object")
        if d.get("type") != "attention":
            raise ConfigError(f"{where}: 'type' must be attention, got {d.get('type')!r}")
        mlp = _obj(d, "mlp", where, optional=True)
        return cls(attention=KeyValueAttentionConfig.from_dict(_obj(d, "mixer", where), where + ".mixer"),
                   mlp=PlainExpertsConfig.from_dict(mlp, where + ".mlp") if mlp is not None else None)

    def to_dict(self) -> dict:
        return {"type": "attention", "mixer": self.attention.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None}


@dataclass(frozen=True)
class FanopelConfig:
    vocab: int
    width: int
    layers: Tuple[FanopelLayer, ...]
    norm_eps: float
    max_positions: int
    residual_mult: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, d: dict, where: str = "config.json") -> "FanopelConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        cfg = cls(vocab=_need(d, "vocab", int, where), width=_need(d, "width", int, where),
                  layers=tuple(FanopelLayer.from_dict(x, f"{where}: layers[{i}]") for i, x in enumerate(layers)),
                  norm_eps=_need(_obj(d, "norm", where), "eps", float, where + ".norm"),
                  max_positions=_need(d, "max_positions", int, where),
                  residual_mult=_typed(d, "residual_mult", float, where) if d.get("residual_mult") is not None else 1.0)
        if cfg.vocab <= 0 or cfg.width <= 0 or cfg.max_positions <= 0:
            raise ConfigError(f"{where}: vocab, width and max_positions must be positive")
        return cfg

    def param_count(self) -> int:
        from ..models.fanopel import fanopel_manifest
        total = 0
        for spec in fanopel_manifest(self).values():
            n = 1
            for x in spec.shape:
                n *= max(int(x), 0)
            total += n
        return total

    def to_dict(self) -> dict:
        return {"architecture": NAME, "vocab": self.vocab, "width": self.width, "max_positions": self.max_positions,
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "layers": [x.to_dict() for x in self.layers]}

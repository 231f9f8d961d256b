"""Typed configuration of the Retezen decoder, read from config.json.

The file is nested.  Top level: ``architecture`` ("Retezen"), ``vocab``, ``width``, ``max_positions`` (rows of the learned
position table), ``norm.eps``, ``logit_scale`` (absent: 1) and ``layers``, a list in which every entry gives ``type``
("attention"), the sizes and constants of its ``mixer`` and its ``mlp`` (null for a layer without a feed-forward).

  mixer:  heads, kv_heads, dim, vdim, scale, mask (size: the window; pool: positions to a pooled block, absent: none;
          without a mask every earlier key is seen), v_mix (whether the values are mixed with those of the first layer
          that says so)
  mlp:    kind "dense" (ff, limit) or "moe" (expert.ff, router.experts, router.top)

Every size and constant that can differ between two models of the design is read from here and from nowhere else;
what the design fixes (the activations, the kind of router) is written where the plan is made.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional, Union

from ..errors import ConfigError, UnsupportedError
from .json_file import read_config_json
from .kugilix import _of


@dataclass(frozen=True)
class RetezenMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None  # mask.size (None: every earlier key is seen)
    pool: Optional[int] = None  # mask.pool (None: nothing is seen before the window)
    v_mix: bool = False

    def to_dict(self) -> dict:
        d: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                   "v_mix": self.v_mix}
        if self.window is not None:
            d["mask"] = {"size": self.window}
            if self.pool is not None:
                d["mask"]["pool"] = self.pool
        return d


@dataclass(frozen=True)
class RetezenDense:
    ff: int
    limit: float

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class RetezenExperts:
    ff: int
    experts: int
    top: int

    def to_dict(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class RetezenLayer:
    mixer: RetezenMixer
    mlp: Optional[Union[RetezenDense, RetezenExperts]]  # None: no feed-forward

    def to_dict(self) -> dict:
        return {"type": "attention", "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class RetezenConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    layers: tuple  # of RetezenLayer
    logit_scale: float = 1.0
    architecture: str = "Retezen"

    # --------------------------------------------------------------- validation
    def validate(self) -> None:
        for name in ("vocab", "width", "max_positions"):
            if getattr(self, name) <= 0:
                raise ConfigError(f"config.json: {name} must be > 0, found {getattr(self, name)}")
        if not (self.norm_eps >= 0.0):
            raise ConfigError(f"config.json: norm.eps must be >= 0, found {self.norm_eps}")
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        mixed = None  # values per token of the layers that mix theirs: one number for all of them
        for i, layer in enumerate(self.layers):
            m, where = layer.mixer, f"layers[{i}]"
            if m.heads <= 0 or m.dim <= 0 or m.vdim <= 0:
                raise ConfigError(f"config.json: {where}.mixer sizes must be > 0")
            if m.kv_heads <= 0 or m.heads % m.kv_heads:
                raise ConfigError(f"config.json: {where}: {m.heads} heads cannot share {m.kv_heads} kv heads")
            if m.window is not None and m.window <= 0:
                raise ConfigError(f"config.json: {where}.mixer.mask.size must be > 0")
            if m.pool is not None and (m.pool <= 0 or m.window is None):
                raise ConfigError(f"config.json: {where}.mixer.mask.pool must be > 0 and stand beside a size")
            if m.v_mix:
                if mixed is None:
                    mixed = m.kv_heads * m.vdim
                elif mixed != m.kv_heads * m.vdim:
                    raise ConfigError(f"config.json: {where}: values of {m.kv_heads} x {m.vdim} cannot be mixed with the {mixed} "
                                      "of the first mixing layer")
            if isinstance(layer.mlp, RetezenDense):
                if layer.mlp.ff <= 0 or not (layer.mlp.limit > 0.0):
                    raise ConfigError(f"config.json: {where}.mlp: ff = {layer.mlp.ff}, limit = {layer.mlp.limit}")
            elif layer.mlp is not None:
                e = layer.mlp
                if e.ff <= 0 or e.experts <= 0 or not (1 <= e.top <= e.experts):
                    raise ConfigError(f"config.json: {where}.mlp: ff = {e.ff}, {e.top} of {e.experts} experts")

    # --------------------------------------------------------------------- I/O
    @classmethod
    def from_dict(cls, d: dict) -> "RetezenConfig":
        name = d.get("architecture") or (d.get("architectures") or [None])[0]
        if name != "Retezen":
            raise UnsupportedError(f"architecture {name!r} is not read by RetezenConfig")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list):
            raise ConfigError("config.json: 'layers' must be a list")
        layers = []
        for i, e in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(e, dict) or not isinstance(e.get("type"), str):
                raise ConfigError(f"config.json: {where} must be an object with a 'type'")
            if e["type"] != "attention":
                raise UnsupportedError(f"config.json: {where}.type '{e['type']}' is not a mixer of this design")
            m = _of(e, "mixer", dict, where)
            mw = where + ".mixer"
            heads, dim = _of(m, "heads", int, mw), _of(m, "dim", int, mw)
            mask = _of(m, "mask", dict, mw, required=False)
            mixer = RetezenMixer(
                heads, _of(m, "kv_heads", int, mw, default=heads, required=False), dim,
                _of(m, "vdim", int, mw, default=dim, required=False), _of(m, "scale", float, mw),
                window=None if mask is None else _of(mask, "size", int, mw + ".mask"),
                pool=None if mask is None else _of(mask, "pool", int, mw + ".mask", required=False),
                v_mix=_of(m, "v_mix", bool, mw, default=False, required=False))
            layers.append(RetezenLayer(mixer, cls._mlp(e.get("mlp"), where + ".mlp")))
        norm = _of(d, "norm", dict, "the top level")
        cfg = cls(
            vocab=_of(d, "vocab", int, "the top level"),
            width=_of(d, "width", int, "the top level"),
            max_positions=_of(d, "max_positions", int, "the top level"),
            norm_eps=_of(norm, "eps", float, "norm"),
            layers=tuple(layers),
            logit_scale=_of(d, "logit_scale", float, "the top level", default=1.0, required=False),
        )
        cfg.validate()
        return cfg

    @staticmethod
    def _mlp(mlp, where):
        if mlp is None:
            return None
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            return RetezenDense(_of(mlp, "ff", int, where), _of(mlp, "limit", float, where))
        if kind == "moe":
            router = _of(mlp, "router", dict, where)
            return RetezenExperts(_of(_of(mlp, "expert", dict, where), "ff", int, where + ".expert"),
                                  _of(router, "experts", int, where + ".router"), _of(router, "top", int, where + ".router"))
        raise UnsupportedError(f"config.json: {where} must be null, of kind 'dense' or of kind 'moe'")

    def to_dict(self) -> dict[str, Any]:
        return {
            "architecture": self.architecture,
            "vocab": self.vocab,
            "width": self.width,
            "max_positions": self.max_positions,
            "norm": {"eps": self.norm_eps},
            "logit_scale": self.logit_scale,
            "layers": [layer.to_dict() for layer in self.layers],
        }

    @classmethod
    def from_json(cls, path: str) -> "RetezenConfig":
        return cls.from_dict(read_config_json(path))

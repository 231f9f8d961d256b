"""Typed configuration of the Lukelorn decoder, read from config.json.

The file is nested.  Top level: ``architecture`` ("Lukelorn"), ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` (the factor
on what every layer adds; absent: 1) and ``layers``, a list in which every entry gives ``type`` (its mixer), the sizes and
constants of its ``mixer``, its ``mlp`` (null for a layer without a feed-forward) and, where it runs another layer's tensors
once more, ``weights_of`` (that layer's index; the rest of the entry then equals that layer's).

  attention:         heads, kv_heads, dim, vdim, scale, softcap, rot, mask (size: the window; keep_first: the first tokens that
                     stay visible; absent: every earlier key is seen)
  latent_attention:  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, mask (size)
  channel_delta:     heads, kv_heads, dim, vdim, conv (taps)
  rot:               base, dims, scaling (factor, low, high, original; absent: none)
  mlp:               kind "dense" (ff) or "moe" (expert.ff, router.experts, router.top)

Every size and constant that can differ between two models of the design is read from here and from nowhere else (the inner
sizes of the recurrence's low-rank projections are those of its tensors); what the design fixes (the activations, the kind of
router, the pairs that rotate together) is written where the plan is made.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional, Union

from ..errors import ConfigError, UnsupportedError
from .json_file import read_config_json
from .kugilix import _of

MIXER_TYPES = ("attention", "latent_attention", "channel_delta")


@dataclass(frozen=True)
class RotaryScaling:
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: Optional[RotaryScaling] = None

    def to_dict(self) -> dict:
        d: dict = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d

    def validate(self, size: int, where: str) -> None:
        if self.dims < 0 or self.dims % 2 or self.dims > size:
            raise ConfigError(f"config.json: {where}: {self.dims} of {size} dimensions rotate")
        if not self.base > 0.0:
            raise ConfigError(f"config.json: {where}.base must be > 0")
        s = self.scaling
        if s is not None and not (s.factor > 0.0 and s.low > 0.0 and s.high > 0.0 and s.original > 0.0):
            raise ConfigError(f"config.json: {where}.scaling: positive numbers are needed")

    @classmethod
    def read(cls, m: dict, default_dims: int, where: str) -> "Rotary":
        rot = _of(m, "rot", dict, where, required=False)
        if rot is None:
            return cls(10000.0, 0)
        where += ".rot"
        scaling = _of(rot, "scaling", dict, where, required=False)
        if scaling is not None:
            scaling = RotaryScaling(*(_of(scaling, k, float, where + ".scaling") for k in ("factor", "low", "high", "original")))
        return cls(_of(rot, "base", float, where), _of(rot, "dims", int, where, default=default_dims, required=False), scaling)


def _positive(obj, names, where: str) -> None:
    for name in names:
        if getattr(obj, name) <= 0:
            raise ConfigError(f"config.json: {where}.{name} must be > 0, found {getattr(obj, name)}")


def _grouped(heads: int, kv_heads: int, where: str) -> None:
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {kv_heads} kv heads")


def _window(m: dict, where: str) -> tuple:
    mask = _of(m, "mask", dict, where, required=False)
    if mask is None:
        return None, 0
    return (_of(mask, "size", int, where + ".mask", required=False),
            _of(mask, "keep_first", int, where + ".mask", default=0, required=False))


@dataclass(frozen=True)
class LukelornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotary
    softcap: Optional[float] = None
    window: Optional[int] = None  # mask.size (None: every earlier key is seen)
    keep_first: int = 0

    def to_dict(self) -> dict:
        d: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot.dims:
            d["rot"] = self.rot.to_dict()
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.window is not None:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return d

    def validate(self, where: str) -> None:
        _positive(self, ("heads", "kv_heads", "dim", "vdim"), where)
        _grouped(self.heads, self.kv_heads, where)
        self.rot.validate(self.dim, where + ".rot")
        if self.softcap is not None and not self.softcap > 0.0:
            raise ConfigError(f"config.json: {where}.softcap must be > 0")
        if self.window is not None and self.window <= 0:
            raise ConfigError(f"config.json: {where}.mask.size must be > 0")
        if self.keep_first < 0:
            raise ConfigError(f"config.json: {where}.mask.keep_first must be >= 0")

    @classmethod
    def read(cls, m: dict, where: str) -> "LukelornAttention":
        heads, dim = _of(m, "heads", int, where), _of(m, "dim", int, where)
        window, keep = _window(m, where)
        return cls(heads, _of(m, "kv_heads", int, where, default=heads, required=False), dim,
                   _of(m, "vdim", int, where, default=dim, required=False), _of(m, "scale", float, where),
                   Rotary.read(m, dim, where), _of(m, "softcap", float, where, required=False), window,
                   0 if window is None else keep)  # without a window every token is seen anyway


@dataclass(frozen=True)
class LukelornLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotary
    window: Optional[int] = None

    def to_dict(self) -> dict:
        d: dict = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                   "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot.dims:
            d["rot"] = self.rot.to_dict()
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d

    def validate(self, where: str) -> None:
        _positive(self, ("heads", "dim", "vdim", "q_rank", "kv_rank"), where)
        if self.rot_dim < 0:
            raise ConfigError(f"config.json: {where}.rot_dim must be >= 0")
        self.rot.validate(self.rot_dim, where + ".rot")
        if self.rot.scaling is not None:
            raise UnsupportedError(f"config.json: {where}.rot.scaling does not belong to this mixer")
        if self.window is not None and self.window <= 0:
            raise ConfigError(f"config.json: {where}.mask.size must be > 0")

    @classmethod
    def read(cls, m: dict, where: str) -> "LukelornLatent":
        rot_dim = _of(m, "rot_dim", int, where, default=0, required=False)
        sizes = [_of(m, k, int, where) for k in ("vdim", "q_rank", "kv_rank")]
        window, keep = _window(m, where)
        if keep:
            raise UnsupportedError(f"config.json: {where}.mask.keep_first does not belong to this mixer")
        return cls(_of(m, "heads", int, where), _of(m, "dim", int, where), rot_dim, *sizes, _of(m, "scale", float, where),
                   Rotary.read(m, rot_dim, where), window)


@dataclass(frozen=True)
class LukelornDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}

    def validate(self, where: str) -> None:
        _positive(self, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
        _grouped(self.heads, self.kv_heads, where)

    @classmethod
    def read(cls, m: dict, where: str) -> "LukelornDelta":
        heads = _of(m, "heads", int, where)
        return cls(heads, _of(m, "kv_heads", int, where, default=heads, required=False), _of(m, "dim", int, where),
                   _of(m, "vdim", int, where), _of(m, "conv", int, where))


_MIXERS = {"attention": LukelornAttention, "latent_attention": LukelornLatent, "channel_delta": LukelornDelta}


@dataclass(frozen=True)
class LukelornDense:
    ff: int

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class LukelornExperts:
    ff: int
    experts: int
    top: int

    def to_dict(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class LukelornLayer:
    type: str  # one of MIXER_TYPES
    mixer: Any  # the sizes class of its type
    mlp: Optional[Union[LukelornDense, LukelornExperts]]  # None: no feed-forward
    weights_of: Optional[int] = None  # the layer whose tensors this one runs once more

    def to_dict(self) -> dict:
        d = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}
        if self.weights_of is not None:
            d["weights_of"] = self.weights_of
        return d


@dataclass(frozen=True)
class LukelornConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple  # of LukelornLayer
    residual_mult: float = 1.0
    architecture: str = "Lukelorn"

    # --------------------------------------------------------------- validation
    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` runs: itself, or the one that ``weights_of`` leads to."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            j = self.layers[i].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ConfigError(f"config.json: layers[{i}].weights_of = {j} leads to no layer with tensors of its own")
            seen.add(j)
            i = j
        return i

    def validate(self) -> None:
        _positive(self, ("vocab", "width"), "the top level")
        if not (self.norm_eps >= 0.0):
            raise ConfigError(f"config.json: norm.eps must be >= 0, found {self.norm_eps}")
        if not (self.residual_mult > 0.0):
            raise ConfigError(f"config.json: residual_mult must be > 0, found {self.residual_mult}")
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            layer.mixer.validate(where + ".mixer")
            e = layer.mlp
            if isinstance(e, LukelornDense) and e.ff <= 0:
                raise ConfigError(f"config.json: {where}.mlp.ff must be > 0")
            if isinstance(e, LukelornExperts) and (e.ff <= 0 or e.experts <= 0 or not (1 <= e.top <= e.experts)):
                raise ConfigError(f"config.json: {where}.mlp: ff = {e.ff}, {e.top} of {e.experts} experts")
            j = self.owner(i)
            if j != i and (layer.type, layer.mixer, layer.mlp) != (self.layers[j].type, self.layers[j].mixer, self.layers[j].mlp):
                raise ConfigError(f"config.json: {where} runs the tensors of layers[{j}] but its entry differs from that one's")

    # --------------------------------------------------------------------- I/O
    @classmethod
    def from_dict(cls, d: dict) -> "LukelornConfig":
        name = d.get("architecture") or (d.get("architectures") or [None])[0]
        if name != "Lukelorn":
            raise UnsupportedError(f"architecture {name!r} is not read by LukelornConfig")
        raw = d.get("layers")
        if not isinstance(raw, list):
            raise ConfigError("config.json: 'layers' must be a list")
        layers = []
        for i, e in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(e, dict) or not isinstance(e.get("type"), str):
                raise ConfigError(f"config.json: {where} must be an object with a 'type'")
            if e["type"] not in _MIXERS:
                raise UnsupportedError(f"config.json: {where}.type '{e['type']}' is not a mixer of this design "
                                       f"({', '.join(MIXER_TYPES)})")
            layers.append(LukelornLayer(
                e["type"], _MIXERS[e["type"]].read(_of(e, "mixer", dict, where), where + ".mixer"),
                cls._mlp(e.get("mlp"), where + ".mlp"), _of(e, "weights_of", int, where, required=False)))
        norm = _of(d, "norm", dict, "the top level")
        cfg = cls(
            vocab=_of(d, "vocab", int, "the top level"),
            width=_of(d, "width", int, "the top level"),
            norm_eps=_of(norm, "eps", float, "norm"),
            layers=tuple(layers),
            residual_mult=_of(d, "residual_mult", float, "the top level", default=1.0, required=False),
        )
        cfg.validate()
        return cfg

    @staticmethod
    def _mlp(mlp, where):
        if mlp is None:
            return None
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            return LukelornDense(_of(mlp, "ff", int, where))
        if kind == "moe":
            router = _of(mlp, "router", dict, where)
            return LukelornExperts(_of(_of(mlp, "expert", dict, where), "ff", int, where + ".expert"),
                                   _of(router, "experts", int, where + ".router"), _of(router, "top", int, where + ".router"))
        raise UnsupportedError(f"config.json: {where} must be null, of kind 'dense' or of kind 'moe'")

    def to_dict(self) -> dict[str, Any]:
        return {
            "architecture": self.architecture,
            "vocab": self.vocab,
            "width": self.width,
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "layers": [layer.to_dict() for layer in self.layers],
        }

    @classmethod
    def from_json(cls, path: str) -> "LukelornConfig":
        return cls.from_dict(read_config_json(path))

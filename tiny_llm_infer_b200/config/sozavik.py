"""Typed configuration of the Sozavik design, read from its own config.json keys.

config.json carries ``architecture`` (the name), ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` (absent or null:
none) and ``layers``: per layer ``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (its
feed-forward, or null for a layer without one).  Layer types:

``attention``    ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` (absent or null: none), ``mask.size``
                 (absent: every key before), ``rot.base``, ``rot.dims`` and ``rot.scaling`` (``factor``, ``low``, ``high``,
                 ``original``; absent or null: none; no ``rot``: no rotation), ``v_mix``.
``attention_2``  ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``, ``v_mix``.
``lightning``    ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head).

Feed-forward ``dense``: ``ff``.  Layers with ``v_mix`` share their value sizes: the first one's values are mixed into the
others'.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple, Union

from .base import ConfigError, ModelConfig, coerce, optional, require

ARCHITECTURE = "Sozavik"


def _section(raw: Dict[str, Any], key: str, where: str, needed: bool = True) -> Optional[Dict[str, Any]]:
    value = raw.get(key)
    if value is None:
        if needed:
            raise ConfigError(f"config.json: {where}{key!r} is missing")
        return None
    if not isinstance(value, dict):
        raise ConfigError(f"config.json: {where}{key!r} must be an object")
    return value


def _positive(obj, names, where: str) -> None:
    for name in names:
        if not getattr(obj, name) > 0:
            raise ConfigError(f"config.json: {where}{name} must be positive")


def _window(raw: Dict[str, Any], where: str) -> Optional[int]:
    mask = _section(raw, "mask", where, needed=False)
    return None if mask is None or mask.get("size") is None else require(mask, "size")


def _softcap(raw: Dict[str, Any], key: str, where: str) -> Optional[float]:
    return None if not raw.get(key) else coerce(raw[key], where + key, float)


def _validate_heads(m, where: str) -> None:
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if m.heads % m.kv_heads:
        raise ConfigError(f"config.json: {where}heads must be a multiple of kv_heads")
    if m.window is not None and m.window <= 0:
        raise ConfigError(f"config.json: {where}mask.size must be positive")


@dataclass(frozen=True)
class FrequencyScaling:
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, raw):
        return cls(*(require(raw, k, float) for k in ("factor", "low", "high", "original")))

    def to_dict(self):
        return {"factor": self.factor, "high": self.high, "low": self.low, "original": self.original}


@dataclass(frozen=True)
class RotatedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None
    window: Optional[int] = None
    rot_base: Optional[float] = None
    rot_dims: int = 0
    rot_scaling: Optional[FrequencyScaling] = None
    v_mix: bool = False

    @classmethod
    def from_dict(cls, raw, where):
        heads, dim = require(raw, "heads"), require(raw, "dim")
        rot = _section(raw, "rot", where, needed=False)
        scaling = None if rot is None else _section(rot, "scaling", where + "rot.", needed=False)
        return cls(heads=heads, kv_heads=optional(raw, "kv_heads", heads), dim=dim, vdim=optional(raw, "vdim", dim),
                   scale=require(raw, "scale", float), softcap=_softcap(raw, "softcap", where), window=_window(raw, where),
                   rot_base=None if rot is None else require(rot, "base", float),
                   rot_dims=0 if rot is None else optional(rot, "dims", dim),
                   rot_scaling=None if scaling is None else FrequencyScaling.from_dict(scaling),
                   v_mix=optional(raw, "v_mix", False, bool))

    def to_dict(self):
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "v_mix": self.v_mix,
               "vdim": self.vdim}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        if self.rot_base is not None:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                out["rot"]["scaling"] = self.rot_scaling.to_dict()
        if self.softcap is not None:
            out["softcap"] = self.softcap
        return out

    def validate(self, where):
        _validate_heads(self, where)
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError(f"config.json: {where}softcap must be positive")
        if self.rot_base is not None:
            if not self.rot_base > 0:
                raise ConfigError(f"config.json: {where}rot.base must be positive")
            if self.rot_dims % 2 or not 0 < self.rot_dims <= self.dim:
                raise ConfigError(f"config.json: {where}rot.dims must be even and within dim")
        if self.rot_scaling is not None:
            _positive(self.rot_scaling, ("factor", "low", "high", "original"), where + "rot.scaling.")
            if self.rot_scaling.high < self.rot_scaling.low:
                raise ConfigError(f"config.json: {where}rot.scaling.high lies below low")


@dataclass(frozen=True)
class WholeNormAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None
    v_mix: bool = False

    @classmethod
    def from_dict(cls, raw, where):
        heads, dim = require(raw, "heads"), require(raw, "dim")
        return cls(heads=heads, kv_heads=optional(raw, "kv_heads", heads), dim=dim, vdim=optional(raw, "vdim", dim),
                   scale=require(raw, "scale", float), window=_window(raw, where), v_mix=optional(raw, "v_mix", False, bool))

    def to_dict(self):
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "v_mix": self.v_mix,
               "vdim": self.vdim}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out

    def validate(self, where):
        _validate_heads(self, where)


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, raw, where):
        heads, dim, decay = require(raw, "heads"), require(raw, "dim"), raw.get("decay")
        if not isinstance(decay, (list, tuple)):
            raise ConfigError(f"config.json: {where}decay must be a list of one number per head")
        return cls(heads=heads, dim=dim, vdim=optional(raw, "vdim", dim),
                   decay=tuple(coerce(a, where + "decay[]", float) for a in decay))

    def to_dict(self):
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}

    def validate(self, where):
        _positive(self, ("heads", "dim", "vdim"), where)
        if len(self.decay) != self.heads:
            raise ConfigError(f"config.json: {where}decay has {len(self.decay)} numbers for {self.heads} heads")


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}

    def validate(self, where):
        _positive(self, ("ff",), where)


MIXERS = {"attention": RotatedAttentionConfig, "attention_2": WholeNormAttentionConfig, "lightning": LightningConfig}


@dataclass(frozen=True)
class SozavikLayerConfig:
    type: str
    mixer: Union[RotatedAttentionConfig, WholeNormAttentionConfig, LightningConfig]
    mlp: Optional[DenseConfig] = None


@dataclass(frozen=True)
class SozavikConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[SozavikLayerConfig, ...]
    logit_softcap: Optional[float] = None
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    architecture: str = field(default=ARCHITECTURE)

    MAX_POSITIONS = 1 << 20       # the design has no table that bounds the context; the cache's size does

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return self.MAX_POSITIONS

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "SozavikConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = require(entry, "type", str)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not a mixer of this design {sorted(MIXERS)}")
            mixer = MIXERS[kind].from_dict(_section(entry, "mixer", where), where + "mixer.")
            mlp_raw = _section(entry, "mlp", where, needed=False)
            mlp = None
            if mlp_raw is not None:
                ff_kind = optional(mlp_raw, "kind", "dense", str)
                if ff_kind != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {ff_kind!r} is not 'dense'")
                mlp = DenseConfig(require(mlp_raw, "ff"))
            layers.append(SozavikLayerConfig(kind, mixer, mlp))
        norm = _section(raw, "norm", "")
        eos = raw.get("eos_token_id")
        if eos is None:
            eos_ids: Tuple[int, ...] = ()
        elif isinstance(eos, (list, tuple)):
            eos_ids = tuple(coerce(x, "eos_token_id[]", int) for x in eos)
        else:
            eos_ids = (coerce(eos, "eos_token_id", int),)
        bos = raw.get("bos_token_id")
        return cls(vocab=require(raw, "vocab"), width=require(raw, "width"), norm_eps=require(norm, "eps", float),
                   layers=tuple(layers), logit_softcap=_softcap(raw, "logit_softcap", ""), eos_token_ids=eos_ids,
                   bos_token_id=None if bos is None else coerce(bos, "bos_token_id", int))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {
            "architecture": self.architecture,
            "layers": [{"mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict(), "type": l.type}
                       for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        if self.bos_token_id is not None:
            out["bos_token_id"] = self.bos_token_id
        return out

    def validate(self) -> None:
        _positive(self, ("vocab", "width"), "")
        if not self.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        mixed = None                  # value sizes of the layers that mix
        for i, layer in enumerate(self.layers):
            layer.mixer.validate(f"layers[{i}].mixer.")
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp.")
            if getattr(layer.mixer, "v_mix", False):
                sizes = (layer.mixer.kv_heads, layer.mixer.vdim)
                if mixed is not None and sizes != mixed:
                    raise ConfigError(f"config.json: layers[{i}] mixes values of {sizes} (heads, width) with values of {mixed}")
                mixed = sizes
        for tok in self.eos_token_ids:
            if not 0 <= tok < self.vocab:
                raise ConfigError(f"config.json: eos_token_id {tok} is outside the vocabulary")

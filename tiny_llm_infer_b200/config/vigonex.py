"""Typed configuration of the Vigonex design, read from its own config.json keys.

config.json carries ``architecture`` (the name), ``vocab``, ``width``, ``streams`` (residual streams), ``embedding.scale``,
``norm.eps``, ``logit_scale`` and ``layers``: per layer ``type`` (which mixer), ``mixer`` (its sizes and constants) and
``mlp`` (its feed-forward, or null for a layer without one).  Layer types:

``attention``      differential attention: ``heads``, ``kv_heads``, ``dim`` (of one map's queries and keys), ``vdim``,
                   ``scale``, ``softcap`` (absent or null: none), ``diff``, ``q_temp.coef`` and ``q_temp.every`` (absent:
                   no temperature).
``general_delta``  the delta rule with a removal rate per channel: ``heads``, ``dim``.  The rank of its decay's low-rank
                   projection is the shape of a tensor.

Feed-forward ``dense``: ``ff``.  Feed-forward ``moe``: ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top``,
``router.scale`` and, if there is a shared expert, ``shared.ff`` and ``shared.limit``.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Dict, Optional, Tuple, Union

from .base import ConfigError, ModelConfig, coerce, optional, require

ARCHITECTURE = "Vigonex"


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


def default_rank(width: int) -> int:
    """Rank of the decay's low-rank projection where no checkpoint says it (random weights)."""
    return max(8, width // 32)


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float] = None
    temp_coef: float = 0.0
    temp_every: Optional[int] = None

    @classmethod
    def from_dict(cls, raw, where):
        heads, cap = require(raw, "heads"), raw.get("softcap")
        temp = _section(raw, "q_temp", where, needed=False)
        return cls(heads=heads, kv_heads=optional(raw, "kv_heads", heads), dim=require(raw, "dim"),
                   vdim=optional(raw, "vdim", raw.get("dim")), scale=require(raw, "scale", float),
                   diff=require(raw, "diff", float), softcap=None if not cap else coerce(cap, where + "softcap", float),
                   temp_coef=0.0 if temp is None else require(temp, "coef", float),
                   temp_every=None if temp is None else require(temp, "every"))

    def to_dict(self):
        out = {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
               "vdim": self.vdim}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.temp_every is not None:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return out

    def validate(self, where):
        _positive(self, ("heads", "kv_heads", "dim", "vdim"), where)
        if self.heads % self.kv_heads:
            raise ConfigError(f"config.json: {where}heads must be a multiple of kv_heads")
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError(f"config.json: {where}softcap must be positive")
        if self.temp_every is not None and self.temp_every <= 0:
            raise ConfigError(f"config.json: {where}q_temp.every must be positive")


@dataclass(frozen=True)
class GeneralDeltaConfig:
    heads: int
    dim: int
    # not a key of config.json: the shape of the checkpoint's tensor gives it (``with_tensor_shapes``)
    decay_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, raw, where):
        return cls(heads=require(raw, "heads"), dim=require(raw, "dim"))

    def to_dict(self):
        return {"dim": self.dim, "heads": self.heads}

    def validate(self, where):
        _positive(self, ("heads", "dim"), where)


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}

    def validate(self, where):
        _positive(self, ("ff",), where)


@dataclass(frozen=True)
class MixtureConfig:
    expert_ff: int
    expert_limit: float
    experts: int
    top: int
    router_scale: float = 1.0
    shared_ff: Optional[int] = None
    shared_limit: Optional[float] = None

    @classmethod
    def from_dict(cls, raw, where):
        expert, router = _section(raw, "expert", where), _section(raw, "router", where)
        shared = _section(raw, "shared", where, needed=False)
        limit = require(expert, "limit", float)
        return cls(expert_ff=require(expert, "ff"), expert_limit=limit, experts=require(router, "experts"),
                   top=require(router, "top"), router_scale=optional(router, "scale", 1.0, float),
                   shared_ff=None if shared is None else require(shared, "ff"),
                   shared_limit=None if shared is None else require(shared, "limit", float))

    def to_dict(self):
        out = {"expert": {"ff": self.expert_ff, "limit": self.expert_limit}, "kind": "moe",
               "router": {"experts": self.experts, "scale": self.router_scale, "top": self.top}}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return out

    def validate(self, where):
        _positive(self, ("expert_ff", "expert_limit", "experts", "top"), where)
        if self.top > self.experts:
            raise ConfigError(f"config.json: {where}router.top exceeds the {self.experts} experts")
        if self.shared_ff is not None:
            _positive(self, ("shared_ff", "shared_limit"), where)


MIXERS = {"attention": DifferentialConfig, "general_delta": GeneralDeltaConfig}


@dataclass(frozen=True)
class VigonexLayerConfig:
    type: str
    mixer: Union[DifferentialConfig, GeneralDeltaConfig]
    mlp: Union[None, DenseConfig, MixtureConfig]


@dataclass(frozen=True)
class VigonexConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[VigonexLayerConfig, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
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
    def from_dict(cls, raw: Dict[str, Any]) -> "VigonexConfig":
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
                if ff_kind == "dense":
                    mlp = DenseConfig(require(mlp_raw, "ff"))
                elif ff_kind == "moe":
                    mlp = MixtureConfig.from_dict(mlp_raw, where + "mlp.")
                else:
                    raise ConfigError(f"config.json: {where}mlp.kind {ff_kind!r} is neither 'dense' nor 'moe'")
            layers.append(VigonexLayerConfig(kind, mixer, mlp))
        embedding = _section(raw, "embedding", "", needed=False) or {}
        norm = _section(raw, "norm", "")
        eos = raw.get("eos_token_id")
        if eos is None:
            eos_ids: Tuple[int, ...] = ()
        elif isinstance(eos, (list, tuple)):
            eos_ids = tuple(coerce(x, "eos_token_id[]", int) for x in eos)
        else:
            eos_ids = (coerce(eos, "eos_token_id", int),)
        bos = raw.get("bos_token_id")
        return cls(vocab=require(raw, "vocab"), width=require(raw, "width"), streams=optional(raw, "streams", 1),
                   norm_eps=require(norm, "eps", float), layers=tuple(layers),
                   embedding_scale=optional(embedding, "scale", 1.0, float),
                   logit_scale=optional(raw, "logit_scale", 1.0, float), eos_token_ids=eos_ids,
                   bos_token_id=None if bos is None else coerce(bos, "bos_token_id", int))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {
            "architecture": self.architecture,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict(), "type": l.type}
                       for l in self.layers],
            "logit_scale": self.logit_scale,
            "norm": {"eps": self.norm_eps},
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        if self.bos_token_id is not None:
            out["bos_token_id"] = self.bos_token_id
        return out

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "VigonexConfig":
        """The sizes that only the checkpoint gives: the ranks of the decays' low-rank projections (rows of
        ``l<i>.mix.w1``)."""
        layers = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, GeneralDeltaConfig):
                w1 = shapes.get(f"l{i}.mix.w1")
                m = replace(m, decay_rank=int(w1[0]) if w1 else m.decay_rank)
            layers.append(replace(layer, mixer=m))
        return replace(self, layers=tuple(layers))

    def validate(self) -> None:
        _positive(self, ("vocab", "width", "streams"), "")
        if not self.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            layer.mixer.validate(f"layers[{i}].mixer.")
            if layer.mlp is not None:
                layer.mlp.validate(f"layers[{i}].mlp.")
        for tok in self.eos_token_ids:
            if not 0 <= tok < self.vocab:
                raise ConfigError(f"config.json: eos_token_id {tok} is outside the vocabulary")

"""Typed configuration of Zinizen, read from its config.json keys.

A Zinizen config.json has ``architecture`` ("Zinizen"), ``vocab``, ``width``, ``norm.eps``, an
optional ``embedding`` (``bigram``: ``buckets``, ``mul_prev``, ``mul_cur`` of the second table that
the token and the one before it choose a row of) and a list ``layers``. Every layer entry gives its
``type`` (the mixer it has: ``attention``, grouped-query attention with a distance bias;
``latent_attention``, softmax attention over one latent row per token; or ``rglru``, a convolution
over time and a gated linear recurrence per channel), the mixer's sizes under ``mixer`` and its
feed-forward under ``mlp`` (null: none; ``kind`` ``dense``: up, gelu, down; ``moe``: routed experts
with clamped gates and, optionally, a shared one).

Nothing here has a default that stands for a size: a key that the design requires and that is
absent is an error with the key's path.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .base import ConfigError, divisible, positive, positive_int

NAME = "Zinizen"


def _need(data: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(data, Mapping) or key not in data:
        raise ConfigError(f"{where}{key} is missing")
    return data[key]


def _sizes(data, keys, where) -> tuple[int, ...]:
    values = tuple(_need(data, key, where) for key in keys)
    for key, value in zip(keys, values):
        positive_int(where + key, value)
    return values


def _number(data, key, where) -> float:
    value = _need(data, key, where)
    positive(where + key, value)
    return float(value)


@dataclass(frozen=True)
class Bigram:
    """The second table's row: (previous * mul_prev + current * mul_cur) mod buckets."""

    buckets: int
    mul_prev: int
    mul_cur: int

    KEYS = ("buckets", "mul_prev", "mul_cur")

    @classmethod
    def from_dict(cls, data, where):
        _sizes(data, ("buckets",), where)
        values = [_need(data, key, where) for key in cls.KEYS]
        for key, value in zip(cls.KEYS, values):
            if isinstance(value, bool) or not isinstance(value, int) or value < 0:
                raise ConfigError(f"{where}{key} must be a non-negative integer, got {value!r}")
        return cls(*values)

    def to_dict(self):
        return {key: getattr(self, key) for key in self.KEYS}


@dataclass(frozen=True)
class Temperature:
    """Queries times 1 + coef * ln(floor((position + 1) / every) + 1)."""

    coef: float
    every: float

    @classmethod
    def from_dict(cls, data, where):
        coef = _need(data, "coef", where)
        if isinstance(coef, bool) or not isinstance(coef, (int, float)):
            raise ConfigError(f"{where}coef must be a number, got {coef!r}")
        return cls(float(coef), _number(data, "every", where))

    def to_dict(self):
        every = int(self.every) if self.every.is_integer() else self.every
        return {"coef": self.coef, "every": every}


@dataclass(frozen=True)
class AttentionMixer:
    """Query heads, key/value heads, query/key and value sizes of a head, score scale, cap of the
    scores, temperature of the queries, whether the values are mixed with the first such layer's."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None = None
    q_temp: Temperature | None = None
    v_mix: bool = False

    SIZES = ("heads", "kv_heads", "dim", "vdim")

    @classmethod
    def from_dict(cls, data, where):
        sizes = _sizes(data, cls.SIZES, where)
        divisible(where + "heads", data["heads"], where + "kv_heads", data["kv_heads"])
        scale = _number(data, "scale", where)
        softcap = None if data.get("softcap") is None else _number(data, "softcap", where)
        q_temp = data.get("q_temp")
        if q_temp is not None:
            q_temp = Temperature.from_dict(q_temp, where + "q_temp.")
        v_mix = data.get("v_mix") or False
        if not isinstance(v_mix, bool):
            raise ConfigError(f"{where}v_mix must be true or false, got {v_mix!r}")
        return cls(*sizes, scale, softcap, q_temp, v_mix)

    def to_dict(self):
        out = {key: getattr(self, key) for key in self.SIZES}
        out["scale"] = self.scale
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.q_temp is not None:
            out["q_temp"] = self.q_temp.to_dict()
        if self.v_mix:
            out["v_mix"] = True
        return out


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int

    @classmethod
    def from_dict(cls, data, where):
        (dims,) = _sizes(data, ("dims",), where)
        if dims % 2:
            raise ConfigError(f"{where}dims ({dims}) must be even")
        return cls(_number(data, "base", where), dims)

    def to_dict(self):
        return {"base": self.base, "dims": self.dims}


@dataclass(frozen=True)
class LatentMixer:
    """Heads, unrotated and rotated query/key sizes, value size, the queries' and the keys'
    latent sizes, score scale, rotation."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotary

    SIZES = ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")

    @classmethod
    def from_dict(cls, data, where):
        sizes = _sizes(data, cls.SIZES, where)
        rot = Rotary.from_dict(_need(data, "rot", where), where + "rot.")
        if rot.dims > data["rot_dim"]:
            raise ConfigError(f"{where}rot.dims ({rot.dims}) exceeds {where}rot_dim ({data['rot_dim']})")
        return cls(*sizes, _number(data, "scale", where), rot)

    def to_dict(self):
        out = {key: getattr(self, key) for key in self.SIZES}
        out.update(rot=self.rot.to_dict(), scale=self.scale)
        return out


@dataclass(frozen=True)
class RecurrentMixer:
    """Width of the two branches, equal parts of the gates' matrices, taps of the convolution."""

    width: int
    blocks: int
    conv: int

    SIZES = ("width", "blocks", "conv")

    @classmethod
    def from_dict(cls, data, where):
        sizes = _sizes(data, cls.SIZES, where)
        divisible(where + "width", data["width"], where + "blocks", data["blocks"])
        return cls(*sizes)

    def to_dict(self):
        return {key: getattr(self, key) for key in self.SIZES}


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int

    @classmethod
    def from_dict(cls, data, where):
        return cls(*_sizes(data, ("ff",), where))

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class Expert:
    """Width of a feed-forward and the limit that its gate and up values are cut at."""

    ff: int
    limit: float

    @classmethod
    def from_dict(cls, data, where):
        (ff,) = _sizes(data, ("ff",), where)
        return cls(ff, _number(data, "limit", where))

    def to_dict(self):
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class RoutedFeedForward:
    """``experts`` feed-forwards of which a token uses ``top``, with weights times ``scale``, and
    a shared one that every token uses (None: there is none)."""

    expert: Expert
    experts: int
    top: int
    scale: float
    shared: Expert | None = None

    @classmethod
    def from_dict(cls, data, where):
        expert = Expert.from_dict(_need(data, "expert", where), where + "expert.")
        router, at = _need(data, "router", where), where + "router."
        experts, top = _sizes(router, ("experts", "top"), at)
        if top > experts:
            raise ConfigError(f"{at}top ({top}) exceeds {at}experts ({experts})")
        scale = 1.0 if router.get("scale") is None else _number(router, "scale", at)
        shared = data.get("shared")
        if shared is not None:
            shared = Expert.from_dict(shared, where + "shared.")
        return cls(expert, experts, top, scale, shared)

    def to_dict(self):
        out = {"expert": self.expert.to_dict(), "kind": "moe",
               "router": {"experts": self.experts, "scale": self.scale, "top": self.top}}
        if self.shared is not None:
            out["shared"] = self.shared.to_dict()
        return out


MIXERS = {"attention": AttentionMixer, "latent_attention": LatentMixer, "rglru": RecurrentMixer}
FEED_FORWARDS = {"dense": DenseFeedForward, "moe": RoutedFeedForward}


@dataclass(frozen=True)
class ZinizenLayer:
    type: str
    mixer: Any                      # AttentionMixer, LatentMixer or RecurrentMixer
    mlp: Any                        # DenseFeedForward, RoutedFeedForward or None

    @classmethod
    def from_dict(cls, data, where):
        kind = _need(data, "type", where)
        if kind not in MIXERS:
            raise ConfigError(f"{where}type {kind!r} is not a mixer of this design "
                              f"({', '.join(sorted(MIXERS))})")
        mixer = MIXERS[kind].from_dict(_need(data, "mixer", where), where + "mixer.")
        mlp = data.get("mlp")
        if mlp is not None:
            form = _need(mlp, "kind", where + "mlp.")
            if form not in FEED_FORWARDS:
                raise ConfigError(f"{where}mlp.kind {form!r} is not known "
                                  f"({', '.join(sorted(FEED_FORWARDS))})")
            mlp = FEED_FORWARDS[form].from_dict(mlp, where + "mlp.")
        return cls(kind, mixer, mlp)

    def to_dict(self):
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": self.type}


@dataclass(frozen=True)
class ZinizenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[ZinizenLayer, ...]
    bigram: Bigram | None = None
    extra: Mapping[str, Any] = field(default_factory=dict, repr=False)

    def __post_init__(self) -> None:
        positive_int("vocab", self.vocab)
        positive_int("width", self.width)
        positive("norm.eps", self.norm_eps)
        if not self.layers:
            raise ConfigError("layers is empty")
        mixed = [(i, layer.mixer) for i, layer in enumerate(self.layers)
                 if isinstance(layer.mixer, AttentionMixer) and layer.mixer.v_mix]
        sizes = lambda mixer: mixer.kv_heads * mixer.vdim
        for i, mixer in mixed[1:]:
            if sizes(mixer) != sizes(mixed[0][1]):
                raise ConfigError(f"layers[{i}].mixer: values of {sizes(mixer)} numbers a token cannot be "
                                  f"mixed with those of layer {mixed[0][0]} ({sizes(mixed[0][1])})")

    @property
    def first_mixed(self) -> int | None:
        """The first layer whose values later layers mix theirs with."""
        for i, layer in enumerate(self.layers):
            if isinstance(layer.mixer, AttentionMixer) and layer.mixer.v_mix:
                return i
        return None

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "ZinizenConfig":
        name = data.get("architecture", data.get("model_type"))
        if str(name).lower() != NAME.lower():
            raise ConfigError(f"architecture {name!r} is not a {NAME} configuration")
        layers = _need(data, "layers", "")
        if not isinstance(layers, (list, tuple)):
            raise ConfigError("layers must be a list")
        bigram = (data.get("embedding") or {}).get("bigram")
        if bigram is not None:
            bigram = Bigram.from_dict(bigram, "embedding.bigram.")
        known = {"architecture", "model_type", "embedding", "layers", "norm", "vocab", "width"}
        return cls(vocab=_need(data, "vocab", ""), width=_need(data, "width", ""),
                   norm_eps=float(_need(_need(data, "norm", ""), "eps", "norm.")),
                   layers=tuple(ZinizenLayer.from_dict(entry, f"layers[{i}].")
                                for i, entry in enumerate(layers)),
                   bigram=bigram, extra={k: v for k, v in data.items() if k not in known})

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = dict(self.extra)
        out.update(architecture=NAME, layers=[layer.to_dict() for layer in self.layers],
                   norm={"eps": self.norm_eps}, vocab=self.vocab, width=self.width)
        if self.bigram is not None:
            out["embedding"] = {"bigram": self.bigram.to_dict()}
        return out

"""Typed configuration of Susalorn, read from its config.json keys.

A Susalorn config.json has ``architecture`` ("Susalorn"), ``vocab``, ``width``, ``norm.eps``,
``streams`` (how many residual streams the layers are connected by), a list ``layers`` and an
optional ``loop``. Every layer entry gives its ``type`` (the mixer it has: ``latent_attention``,
softmax attention over one latent row per token whose queries go through a latent too, with
YaRN-scaled rotary positions and a sink per head; or ``channel_delta``, the gated delta rule with
a decay per key channel), the mixer's sizes under ``mixer`` and its feed-forward under ``mlp``
(null: none; ``kind`` ``dense``: a gated feed-forward; ``moe``: routed experts without gates).
``loop`` names a run of layers (``start`` .. ``stop`` - 1) that is executed ``times`` times in a
row with the same weights.

Two inner sizes of ``channel_delta`` are not in the file: the stored tensors decide them. A
configuration for random weights may name them (``decay_rank``, ``gate_rank``).

Nothing here has a default that stands for a size: a key that the design requires and that is
absent is an error with the key's path.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .base import ConfigError, divisible, positive, positive_int

NAME = "Susalorn"


def _need(data: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(data, Mapping) or key not in data:
        raise ConfigError(f"{where}{key} is missing")
    return data[key]


def _sizes(data, keys, where) -> tuple[int, ...]:
    values = tuple(_need(data, key, where) for key in keys)
    for key, value in zip(keys, values):
        positive_int(where + key, value)
    return values


@dataclass(frozen=True)
class FrequencyScaling:
    """YaRN: rotary frequencies for a context ``factor`` times the ``original`` one; pairs that
    turn ``fast`` times or more within it keep theirs, pairs that turn ``slow`` times or less are
    divided by ``factor``."""

    factor: float
    fast: float
    slow: float
    original: float

    KEYS = ("factor", "fast", "slow", "original")

    @classmethod
    def from_dict(cls, data, where):
        values = [_need(data, key, where) for key in cls.KEYS]
        for key, value in zip(cls.KEYS, values):
            positive(where + key, value)
        return cls(*(float(value) for value in values))

    def to_dict(self):
        original = int(self.original) if float(self.original).is_integer() else self.original
        return {"factor": self.factor, "fast": self.fast, "original": original, "slow": self.slow}


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int
    scaling: FrequencyScaling | None = None

    @classmethod
    def from_dict(cls, data, where):
        (dims,) = _sizes(data, ("dims",), where)
        if dims % 2:
            raise ConfigError(f"{where}dims ({dims}) must be even")
        base = _need(data, "base", where)
        positive(where + "base", base)
        scaling = data.get("scaling")
        if scaling is not None and base == 1:
            raise ConfigError(f"{where}base must not be 1 where frequencies are scaled")
        return cls(float(base), dims, None if scaling is None
                   else FrequencyScaling.from_dict(scaling, where + "scaling."))

    def to_dict(self):
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = self.scaling.to_dict()
        return out


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
        scale = _need(data, "scale", where)
        positive(where + "scale", scale)
        rot = Rotary.from_dict(_need(data, "rot", where), where + "rot.")
        if rot.dims > data["rot_dim"]:
            raise ConfigError(f"{where}rot.dims ({rot.dims}) exceeds {where}rot_dim ({data['rot_dim']})")
        return cls(*sizes, float(scale), rot)

    def to_dict(self):
        out = {key: getattr(self, key) for key in self.SIZES}
        out.update(rot=self.rot.to_dict(), scale=self.scale)
        return out


@dataclass(frozen=True)
class ChannelDeltaMixer:
    """Value heads, query/key heads, key and value sizes, taps of the convolutions; the inner
    sizes of the decay's and the gate's projections, where the configuration names them."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int | None = None
    gate_rank: int | None = None

    SIZES = ("heads", "kv_heads", "dim", "vdim", "conv")
    RANKS = ("decay_rank", "gate_rank")

    @classmethod
    def from_dict(cls, data, where):
        sizes = _sizes(data, cls.SIZES, where)
        divisible(where + "heads", data["heads"], where + "kv_heads", data["kv_heads"])
        ranks = [data.get(key) for key in cls.RANKS]
        for key, value in zip(cls.RANKS, ranks):
            if value is not None:
                positive_int(where + key, value)
        return cls(*sizes, *ranks)

    def to_dict(self):
        out = {key: getattr(self, key) for key in self.SIZES}
        out.update({key: getattr(self, key) for key in self.RANKS if getattr(self, key) is not None})
        return out


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int

    @classmethod
    def from_dict(cls, data, where):
        return cls(*_sizes(data, ("ff",), where))

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class RoutedFeedForward:
    """``experts`` feed-forwards of width ``ff`` of which a token uses ``top``, with weights
    times ``scale``; experts form ``groups`` equal runs of neighbours of which the best ``keep``
    may be chosen from."""

    ff: int
    experts: int
    top: int
    groups: int
    keep: int
    scale: float

    @classmethod
    def from_dict(cls, data, where):
        (ff,) = _sizes(_need(data, "expert", where), ("ff",), where + "expert.")
        router, at = _need(data, "router", where), where + "router."
        experts, top = _sizes(router, ("experts", "top"), at)
        groups, keep = 1, 1
        if router.get("groups") is not None:
            groups, keep = _sizes(router["groups"], ("count", "keep"), at + "groups.")
            divisible(at + "experts", experts, at + "groups.count", groups)
            if keep > groups:
                raise ConfigError(f"{at}groups.keep ({keep}) exceeds {at}groups.count ({groups})")
        if top > keep * (experts // groups):
            raise ConfigError(f"{at}top ({top}) exceeds the experts of the kept groups")
        scale = router.get("scale", 1.0)
        positive(at + "scale", scale)
        return cls(ff, experts, top, groups, keep, float(scale))

    def to_dict(self):
        return {"expert": {"ff": self.ff}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep},
                           "scale": self.scale, "top": self.top}}


MIXERS = {"latent_attention": LatentMixer, "channel_delta": ChannelDeltaMixer}
FEED_FORWARDS = {"dense": DenseFeedForward, "moe": RoutedFeedForward}


@dataclass(frozen=True)
class SusalornLayer:
    type: str
    mixer: Any                      # LatentMixer or ChannelDeltaMixer
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
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class SusalornConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int
    layers: tuple[SusalornLayer, ...]
    loop: Loop | None = None
    extra: Mapping[str, Any] = field(default_factory=dict, repr=False)

    def __post_init__(self) -> None:
        positive_int("vocab", self.vocab)
        positive_int("width", self.width)
        positive_int("streams", self.streams)
        positive("norm.eps", self.norm_eps)
        if not self.layers:
            raise ConfigError("layers is empty")
        if self.loop is not None:
            loop = self.loop
            for key in ("start", "stop", "times"):
                value = getattr(loop, key)
                if isinstance(value, bool) or not isinstance(value, int) or value < 0:
                    raise ConfigError(f"loop.{key} must be a non-negative integer, got {value!r}")
            if not loop.start < loop.stop <= len(self.layers):
                raise ConfigError(f"loop.start .. loop.stop ({loop.start} .. {loop.stop}) is not "
                                  f"a run of the {len(self.layers)} layers")
            positive_int("loop.times", loop.times)

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "SusalornConfig":
        name = data.get("architecture", data.get("model_type"))
        if str(name).lower() != NAME.lower():
            raise ConfigError(f"architecture {name!r} is not a {NAME} configuration")
        layers = _need(data, "layers", "")
        if not isinstance(layers, (list, tuple)):
            raise ConfigError("layers must be a list")
        loop = data.get("loop")
        if loop is not None:
            loop = Loop(*(_need(loop, key, "loop.") for key in ("start", "stop", "times")))
        known = {"architecture", "model_type", "layers", "loop", "norm", "streams", "vocab", "width"}
        return cls(vocab=_need(data, "vocab", ""), width=_need(data, "width", ""),
                   norm_eps=float(_need(_need(data, "norm", ""), "eps", "norm.")),
                   streams=_need(data, "streams", ""),
                   layers=tuple(SusalornLayer.from_dict(entry, f"layers[{i}].")
                                for i, entry in enumerate(layers)),
                   loop=loop, extra={k: v for k, v in data.items() if k not in known})

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = dict(self.extra)
        out.update(architecture=NAME, layers=[layer.to_dict() for layer in self.layers],
                   norm={"eps": self.norm_eps}, streams=self.streams, vocab=self.vocab,
                   width=self.width)
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop,
                           "times": self.loop.times}
        return out

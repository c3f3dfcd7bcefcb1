"""Susalorn described in parts.

The layers are joined by hyper-connections: several residual streams, all equal to the token's
embedding at the start; a sublayer reads a stored weighting of them, its normed reading goes
through the mixer or feed-forward, and every stream becomes a stored mixture of all streams plus a
multiple of the sublayer's output. After the last layer the streams are added up. The mixer of a
layer is either attention over one latent row per token (queries through a latent of their own, a
rotated key part shared by the heads with YaRN frequencies, a sink per head) or the gated delta
rule with a decay per key channel. The feed-forward is gated (silu), or a mixture of routed
experts down(relu(up x)^2) chosen by softmax scores within the best groups, or absent. A run of
layers may be executed several times with the same weights; each pass has cache entries of its
own. The output matrix is the embedding table.

Stored names: ``embed``, ``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.{in,out,mix}``, ``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,
uv,sink,o}`` (latent attention) or ``l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,a1,a2,A_log,dt_bias,
norm,g1,g2,o}`` (delta rule), ``l<i>.mlp.{gate,up,down}`` (dense) or ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.{up,down}`` (experts); matrices are [out, in].
"""

from __future__ import annotations

from ..config.registry import Architecture
from ..config.susalorn import (ChannelDeltaMixer, DenseFeedForward, LatentMixer, RoutedFeedForward,
                               SusalornConfig)
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _latent(mixer: LatentMixer, width: int, eps: float) -> PartSpec:
    scaling = mixer.rot.scaling
    position = PartSpec("yarn", {
        "theta": mixer.rot.base, "rotary_dim": mixer.rot.dims,
        "factor": None if scaling is None else scaling.factor,
        "original": None if scaling is None else scaling.original,
        "fast": None if scaling is None else scaling.fast,
        "slow": None if scaling is None else scaling.slow})
    return PartSpec("latent_attention", {
        "hidden": width, "heads": mixer.heads, "head_dim": mixer.dim, "rot_dim": mixer.rot_dim,
        "value_dim": mixer.vdim, "latent": mixer.kv_rank, "query_latent": mixer.q_rank,
        "eps": eps, "position": position, "scale": mixer.scale, "gate": False, "sink": True,
    }, "mix.", {"query_down": "dq", "query_norm": "dq.norm", "query_up": "uq", "down": "dkv",
                "down_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "out": "o"})


def _delta(mixer: ChannelDeltaMixer, width: int, eps: float) -> PartSpec:
    return PartSpec("channel_delta", {
        "hidden": width, "heads": mixer.heads, "kv_heads": mixer.kv_heads, "key_dim": mixer.dim,
        "value_dim": mixer.vdim, "taps": mixer.conv, "eps": eps,
        "decay_rank": mixer.decay_rank, "gate_rank": mixer.gate_rank}, "mix.")


def _feed_forward(mlp, width: int) -> PartSpec:
    if isinstance(mlp, DenseFeedForward):
        return PartSpec("swiglu", {"hidden": width, "width": mlp.ff}, "mlp.",
                        {"w1.weight": "gate", "w3.weight": "up", "w2.weight": "down"})
    assert isinstance(mlp, RoutedFeedForward)
    return PartSpec("routed", {
        "hidden": width, "width": mlp.ff, "experts": mlp.experts, "top": mlp.top,
        "groups": mlp.groups, "keep": mlp.keep, "group_score": 1, "scale": mlp.scale,
        "scores": "softmax", "gated": False, "activation": "relu2"}, "mlp.")


def call_order(config: SusalornConfig) -> tuple[LayerCall, ...]:
    """The layers in the order they run, a looped run unrolled."""
    count, loop = len(config.layers), config.loop
    order = list(range(count))
    if loop is not None:
        looped = list(range(loop.start, loop.stop))
        order = list(range(loop.start)) + looped * loop.times + list(range(loop.stop, count))
    return tuple(LayerCall(index) for index in order)


def describe(config: SusalornConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = lambda name: PartSpec("rmsnorm", {"size": width, "eps": eps}, "", {"weight": name})
    layers = []
    for index, layer in enumerate(config.layers):
        if isinstance(layer.mixer, LatentMixer):
            mixer = _latent(layer.mixer, width, eps)
        else:
            mixer = _delta(layer.mixer, width, eps)
        feed_forward = feed_forward_norm = None
        if layer.mlp is not None:
            feed_forward = _feed_forward(layer.mlp, width)
            feed_forward_norm = norm("norm2")
        block = PartSpec("hyper", {"streams": config.streams, "feed_forward": layer.mlp is not None},
                         "", {f"{name}{which}": f"hc{which}.{name}"
                              for name in ("in", "out", "mix") for which in (1, 2)})
        layers.append(LayerSpec(prefix=f"l{index}.", block=block, mixer=mixer,
                                mixer_norm=norm("norm1"), feed_forward=feed_forward,
                                feed_forward_norm=feed_forward_norm))
    return ModelSpec(
        architecture="susalorn", vocab_size=config.vocab, hidden_size=width, embedding="embed",
        layers=tuple(layers), order=call_order(config), final_norm=norm("final.norm"), head=None,
        max_positions=1 << 30)


ARCHITECTURE = Architecture("susalorn", SusalornConfig, describe)

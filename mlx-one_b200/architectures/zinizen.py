"""Zinizen described in parts.

The stream starts as the token's row of one table plus a row of a second table that the token and
the one before it choose. Every sublayer is normed ahead of it and behind it (layer norms with
biases). The mixer of a layer is grouped-query attention whose queries and keys are normed over the
whole projection, with a temperature on the queries, capped scores, a bias that falls with the
distance, and values that are mixed with the first such layer's; or attention over one latent row
per token with a gate per head; or a convolution over time followed by a gated linear recurrence
per channel. The feed-forward is dense (gelu), or a mixture of routed experts with clamped gates
beside a shared one, or absent. The output matrix is stored.

Stored names: ``embed``, ``bigram``, ``final.norm``, ``head``, and per layer i ``l<i>.norm1``,
``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b`` (each with its bias under the same name and
``.b``), ``l<i>.mix.{q,k,v,q.norm,k.norm,vmix,o}`` (attention), ``l<i>.mix.{dq,dq.norm,uq,dkv,
dkv.norm,uk,uv,g,o}`` (latent attention) or ``l<i>.mix.{y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,
lam,o}`` (recurrence), ``l<i>.mlp.{up,down}`` (dense) or ``l<i>.mlp.{router,correction}``,
``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down}``; matrices are [out, in].
"""

from __future__ import annotations

from ..config.registry import Architecture
from ..config.zinizen import (AttentionMixer, DenseFeedForward, LatentMixer, RecurrentMixer,
                              RoutedFeedForward, ZinizenConfig)
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _attention(mixer: AttentionMixer, width: int, eps: float, mix: str | None) -> PartSpec:
    heads = mixer.heads
    return PartSpec("attention", {
        "hidden": width, "heads": heads, "kv_heads": mixer.kv_heads, "head_dim": mixer.dim,
        "value_dim": mixer.vdim, "qk_norm_eps": eps, "qk_norm": "weighted_rows",
        "scale": mixer.scale, "score_cap": mixer.softcap,
        "distance_slopes": tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)),
        "temperature": None if mixer.q_temp is None else (mixer.q_temp.coef, mixer.q_temp.every),
        "value_mix": mix,
    }, "mix.", {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v",
                "out_proj.weight": "o", "q_layernorm.weight": "q.norm",
                "k_layernorm.weight": "k.norm", "value_mix": "vmix"})


def _latent(mixer: LatentMixer, width: int, eps: float) -> PartSpec:
    position = PartSpec("yarn", {"theta": mixer.rot.base, "rotary_dim": mixer.rot.dims})
    return PartSpec("latent_attention", {
        "hidden": width, "heads": mixer.heads, "head_dim": mixer.dim, "rot_dim": mixer.rot_dim,
        "value_dim": mixer.vdim, "latent": mixer.kv_rank, "query_latent": mixer.q_rank,
        "eps": eps, "position": position, "scale": mixer.scale, "gate": "heads",
    }, "mix.", {"query_down": "dq", "query_norm": "dq.norm", "query_up": "uq", "down": "dkv",
                "down_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "gate": "g", "out": "o"})


def _recurrence(mixer: RecurrentMixer, width: int) -> PartSpec:
    return PartSpec("rglru", {"hidden": width, "width": mixer.width, "blocks": mixer.blocks,
                              "taps": mixer.conv}, "mix.")


def _feed_forward(mlp, width: int) -> PartSpec:
    if isinstance(mlp, DenseFeedForward):
        return PartSpec("dense", {"hidden": width, "width": mlp.ff, "activation": "gelu_tanh"},
                        "mlp.", {"up.weight": "up", "down.weight": "down"})
    assert isinstance(mlp, RoutedFeedForward)
    return PartSpec("routed", {
        "hidden": width, "width": mlp.expert.ff, "experts": mlp.experts, "top": mlp.top,
        "scale": mlp.scale, "scores": "softmax", "correction": True, "activation": "clamped",
        "limit": mlp.expert.limit, "shared_width": None if mlp.shared is None else mlp.shared.ff,
        "shared_limit": None if mlp.shared is None else mlp.shared.limit}, "mlp.")


def describe(config: ZinizenConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = lambda name: PartSpec("layernorm", {"size": width, "eps": eps}, "",
                                 {"weight": name, "bias": name + ".b"})
    layers = []
    for index, layer in enumerate(config.layers):
        if isinstance(layer.mixer, AttentionMixer):
            mix = None
            if layer.mixer.v_mix:
                mix = "first" if index == config.first_mixed else "later"
            mixer = _attention(layer.mixer, width, eps, mix)
        elif isinstance(layer.mixer, LatentMixer):
            mixer = _latent(layer.mixer, width, eps)
        else:
            mixer = _recurrence(layer.mixer, width)
        feed_forward = feed_forward_norm = None
        if layer.mlp is not None:
            feed_forward = _feed_forward(layer.mlp, width)
            feed_forward_norm = norm("norm2")
        block = PartSpec("sandwich", {"size": width, "eps": eps, "norm": "layernorm",
                                      "feed_forward": layer.mlp is not None}, "",
                         {"post_mixer": "norm1b", "post_mixer.bias": "norm1b.b",
                          "post_feed_forward": "norm2b", "post_feed_forward.bias": "norm2b.b"})
        layers.append(LayerSpec(prefix=f"l{index}.", block=block, mixer=mixer,
                                mixer_norm=norm("norm1"), feed_forward=feed_forward,
                                feed_forward_norm=feed_forward_norm))
    embedding_part = None
    if config.bigram is not None:
        rule = config.bigram
        embedding_part = PartSpec("pair_hash", {
            "vocab": config.vocab, "hidden": width, "buckets": rule.buckets,
            "mul_prev": rule.mul_prev, "mul_cur": rule.mul_cur}, "",
            {"table": "embed", "pairs": "bigram"})
    return ModelSpec(
        architecture="zinizen", vocab_size=config.vocab, hidden_size=width, embedding="embed",
        layers=tuple(layers), order=tuple(LayerCall(index) for index in range(len(layers))),
        final_norm=norm("final.norm"), head="head", max_positions=1 << 30,
        embedding_part=embedding_part)


ARCHITECTURE = Architecture("zinizen", ZinizenConfig, describe)

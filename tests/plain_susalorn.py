"""Plain, slow Susalorn written from the design's equations: whole sequences, no cache, one
function per mechanism. It shares no code with the engine: it reads config.json and the
safetensors file by itself and computes everything in one floating type (float64 by default).

Notation: T tokens at positions 0..T-1; X [S, T, W] the S streams; h [T, W] a sublayer's input.
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

_KINDS = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}


def read_tensors(path):
    """A safetensors file: 8 bytes little-endian header length, the JSON header, the data."""
    raw = Path(path).read_bytes()
    (length,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + length])
    data = raw[8 + length:]
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=_KINDS[info["dtype"]]) \
            .reshape(info["shape"]).clone()
    return out


# --------------------------------------------------------------------------- small pieces


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def read_streams(X, weights):
    """What a sublayer reads: sum_s weights[s] X_s."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + weights[s] * X[s]
    return u


def write_streams(X, mix, out, y):
    """New stream t: sum_s mix[s, t] X_s + out[t] y, all from the old streams."""
    new = torch.zeros_like(X)
    for t in range(X.shape[0]):
        for s in range(X.shape[0]):
            new[t] = new[t] + mix[s, t] * X[s]
        new[t] = new[t] + out[t] * y
    return new


# --------------------------------------------------------------------------- latent attention


def rotation(rot):
    """(frequency of every pair, factor on cosine and sine), YaRN where ``scaling`` is given."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0

    def turning(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turning(scaling["fast"])), 0)
    hi = min(math.ceil(turning(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, heads, R]: dimension i < dims/2 turns with dimension i + dims/2; dimensions from dims
    on pass."""
    dims = rot["dims"]
    freq, factor = rotation(rot)
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(x.dtype) * freq[i]
        cos, sin = (torch.cos(angle) * factor)[:, None], (torch.sin(angle) * factor)[:, None]
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * cos - v * sin
        out[..., i + dims // 2] = v * cos + u * sin
    return out


def softmax_with_sink(scores, mask, sink):
    """Rows of exp(score) / (exp(sink) + sum of exp(score) over the visible keys)."""
    scores = scores.masked_fill(~mask, float("-inf"))
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, w, m, eps, prefix):
    """Queries through a latent of their own; keys and values of all heads from one small latent
    per token; one rotated key part shared by the heads; a sink per head."""
    T = h.shape[0]
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T)
    query_latent = rms_norm(h @ w[prefix + "dq"].T, w[prefix + "dq.norm"], eps)
    q = (query_latent @ w[prefix + "uq"].T).view(T, H, D + R)
    down = h @ w[prefix + "dkv"].T
    latent = rms_norm(down[:, :C], w[prefix + "dkv.norm"], eps)
    q_rot = rotate_halves(q[..., D:], positions, m["rot"])
    k_rot = rotate_halves(down[:, C:].view(T, 1, R), positions, m["rot"])[:, 0]
    k_plain = (latent @ w[prefix + "uk"].T).view(T, H, D)
    v = (latent @ w[prefix + "uv"].T).view(T, H, V)
    mask = torch.arange(T)[:, None] >= torch.arange(T)[None, :]
    heads = []
    for n in range(H):
        scores = (q[:, n, :D] @ k_plain[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]
        heads.append(softmax_with_sink(scores, mask, w[prefix + "sink"][n]) @ v[:, n])
    return torch.cat(heads, -1) @ w[prefix + "o"].T


# --------------------------------------------------------------------------- channel-wise delta rule


def convolve(x, kernel):
    """silu of the causal convolution of every channel, last column the current token's."""
    taps = kernel.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        shifted = torch.zeros_like(x)
        shifted[back:] = x[:x.shape[0] - back] if back else x
        out = out + kernel[:, j] * shifted
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, beta, decay):
    """Per head on S [D, V] from zero: rows of S times the token's decays, then u = beta (v -
    S^T k), S += k u^T, o = S^T q. q, k, decay [T, H, D]; v [T, H, V]; beta [T, H]."""
    T, H, D = q.shape
    out = torch.zeros_like(v)
    S = torch.zeros(H, D, v.shape[2], dtype=v.dtype)
    for t in range(T):
        S = S * decay[t][:, :, None]
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def channel_delta(h, w, m, eps, prefix):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (convolve(h @ w[prefix + n].T, w[prefix + n + ".conv"]) for n in ("q", "k", "v"))
    share = H // G
    q = (unit(q.view(T, G, D)) * D ** -0.5).repeat_interleave(share, 1)
    k = unit(k.view(T, G, D)).repeat_interleave(share, 1)
    beta = torch.sigmoid(h @ w[prefix + "b"].T)
    step = softplus((h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "dt_bias"])
    decay = torch.exp(-torch.exp(w[prefix + "A_log"])[None, :, None] * step.view(T, H, D))
    o = delta_recurrence(q, k, v.view(T, H, V), beta, decay)
    gate = torch.sigmoid((h @ w[prefix + "g1"].T) @ w[prefix + "g2"].T).view(T, H, V)
    return (rms_norm(o, w[prefix + "norm"], eps) * gate).reshape(T, H * V) @ w[prefix + "o"].T


MIXERS = {"latent_attention": latent_attention, "channel_delta": channel_delta}


# --------------------------------------------------------------------------- feed-forwards


def dense(h, w, m, prefix, margins=None):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def route(logits, router, margins=None):
    """Weights [T, experts]: softmax over all experts, the best groups by their largest score, the
    best experts among theirs, normalised and scaled. ``margins``: a list that receives, per
    token, by how much (in logits) the choice of groups and experts was made."""
    T, E = logits.shape
    scores = torch.softmax(logits, -1)
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    out = torch.zeros_like(scores)
    margin = torch.full((T,), float("inf"), dtype=torch.float64)
    for t in range(T):
        best = [max(float(scores[t, g * size + i]) for i in range(size)) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: (-best[g], g))[:groups["keep"]]
        allowed = [e for e in range(E) if e // size in kept]
        chosen = sorted(allowed, key=lambda e: (-float(scores[t, e]), e))[:router["top"]]
        total = sum(scores[t, e] for e in chosen) + 1e-20
        for e in chosen:
            out[t, e] = scores[t, e] / total * router.get("scale", 1.0)
        worst = min(math.log(best[g] + 1e-300) for g in kept)
        for g in range(len(best)):
            if g not in kept:
                margin[t] = min(float(margin[t]), worst - math.log(best[g] + 1e-300))
        worst = min(float(logits[t, e]) for e in chosen)
        for e in allowed:
            if e not in chosen:
                margin[t] = min(float(margin[t]), worst - float(logits[t, e]))
    if margins is not None:
        margins.append(margin)
    return out


def experts(h, w, m, prefix, margins=None):
    weights = route(h @ w[prefix + "router"].T, m["router"], margins)
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        hidden = torch.clamp(h @ w[f"{prefix}e{e}.up"].T, min=0) ** 2
        out = out + weights[:, e:e + 1] * (hidden @ w[f"{prefix}e{e}.down"].T)
    return out


FEED_FORWARDS = {"dense": dense, "moe": experts}


# --------------------------------------------------------------------------- the model


def layer_order(config):
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(count))
    looped = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + looped * loop["times"] + list(range(loop["stop"], count))


def forward(config, weights, tokens, kind=torch.float64, streams=None, margins=None):
    """Logits [T, vocab] of one sequence. ``streams``: a list that receives the sum of the
    streams after the embedding and after every layer run; ``margins``: see ``route``."""
    w = {name: t.to(kind) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = x[None].repeat(config.get("streams", 1), 1, 1)
    if streams is not None:
        streams.append(X.sum(0))
    for i in layer_order(config):
        layer, p = config["layers"][i], f"l{i}."
        h = rms_norm(read_streams(X, w[p + "hc1.in"]), w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, w, layer["mixer"], eps, p + "mix.")
        X = write_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        if layer.get("mlp") is not None:
            h = rms_norm(read_streams(X, w[p + "hc2.in"]), w[p + "norm2"], eps)
            y = FEED_FORWARDS[layer["mlp"]["kind"]](h, w, layer["mlp"], p + "mlp.", margins)
            X = write_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], y)
        if streams is not None:
            streams.append(X.sum(0))
    return rms_norm(X.sum(0), w["final.norm"], eps) @ w["embed"].T


def load(model_dir):
    path = Path(model_dir)
    return json.loads((path / "config.json").read_text()), read_tensors(path / "model.safetensors")

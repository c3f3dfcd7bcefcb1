"""Plain, slow Zinizen written from the design's equations: whole sequences, no cache, one
function per mechanism. It shares no code with the engine: it reads config.json and the
safetensors file by itself and computes everything in one floating type (float64 by default).

Notation: T tokens at positions 0..T-1; x [T, W] the stream; h [T, W] a part's normed input.
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


def layer_norm(x, w, b, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def softmax_rows(scores, visible):
    scores = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def causal(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


# --------------------------------------------------------------------------- embedding


def embedding(w, rule, tokens):
    """Row of the token plus a row of a second table picked by the pair (previous, current)."""
    buckets = rule["buckets"]
    rows = []
    for t, token in enumerate(tokens):
        rows.append(buckets if t == 0 else
                    (int(tokens[t - 1]) * rule["mul_prev"] + int(token) * rule["mul_cur"]) % buckets)
    return w["embed"][torch.as_tensor(tokens, dtype=torch.long)] + w["bigram"][torch.tensor(rows)]


# --------------------------------------------------------------------------- attention


def temperature(positions, rule, kind):
    """The factor on a query: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1 + rule["coef"] * math.log(math.floor((int(p) + 1) / rule["every"]) + 1)
                         for p in positions], dtype=kind)


def slopes(heads, kind):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=kind)


def biased_attention(q, k, v, scale, cap, slope):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: capped scores, then slope_h times the
    distance taken off, a softmax over the keys at and before the query."""
    T, H, _ = q.shape
    G = k.shape[1]
    distance = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        s = s - slope[h] * distance
        out[:, h] = softmax_rows(s, causal(T)) @ v[:, g]
    return out


def mix_values(v, first, factor):
    return (1 - factor) * v + factor * first


def attention(h, w, m, eps, p, shared):
    """``shared``: a dict that lives for one forward pass (it holds the first mixing layer's v)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, D)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, D)
    v = h @ w[p + "v"].T
    if m.get("q_temp"):
        q = q * temperature(range(T), m["q_temp"], q.dtype)[:, None, None]
    if m.get("v_mix"):
        if "values" in shared:
            v = mix_values(v, shared["values"], w[p + "vmix"].reshape(()))
        else:
            shared["values"] = v
    out = biased_attention(q, k, v.view(T, G, V), m["scale"], m.get("softcap"), slopes(H, h.dtype))
    return out.reshape(T, H * V) @ w[p + "o"].T


def rotate_halves(x, rot):
    """x [T, heads, R]: dimension i < dims/2 turns with dimension i + dims/2 by t * f_i."""
    dims, half = rot["dims"], rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None, None] * f
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(angle) - v * torch.sin(angle),
                      v * torch.cos(angle) + u * torch.sin(angle), x[..., dims:]], -1)


def latent_attention(h, w, m, eps, p, shared=None):
    """Queries through a latent of their own; keys and values of all heads from one small latent
    per token; one rotated key part shared by the heads; one gate number per head."""
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    r = rotate_halves(down[:, C:].view(T, 1, R), m["rot"])[:, 0]
    q_rot = rotate_halves(q[..., D:], m["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    heads = []
    for n in range(H):
        s = (q[:, n, :D] @ k[:, n].T + q_rot[:, n] @ r.T) * m["scale"]
        heads.append(softmax_rows(s, causal(T)) @ v[:, n] * gate[:, n:n + 1])
    return torch.cat(heads, -1) @ w[p + "o"].T


# --------------------------------------------------------------------------- gated linear recurrence


def conv_over_time(u, kernel, bias):
    """u [T, C], kernel [C, taps]: the last column weighs the token itself, nothing ahead of the
    sequence's start."""
    T, taps = u.shape[0], kernel.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + T] * kernel[:, j] for j in range(taps)) + bias


def block_products(u, matrices, bias):
    """u [T, C] in as many equal parts as there are matrices [out, in]; each part by its own."""
    count, n = matrices.shape[0], matrices.shape[1]
    parts = [u[:, b * n:(b + 1) * n] @ matrices[b].T + bias[b] for b in range(count)]
    return torch.cat(parts, -1)


def linear_recurrence(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t, a_t = exp(-8 r_t softplus(lam)), from zero."""
    out = torch.zeros_like(u)
    S = torch.zeros_like(u[0])
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru(h, w, m, eps, p, shared=None):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = conv_over_time(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_products(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_products(u, w[p + "ri"], w[p + "ri.b"]))
    return (linear_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "rglru": rglru}


# --------------------------------------------------------------------------- feed-forwards


def dense(h, w, m, p, margins=None):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def clamped_unit(h, w, limit, p):
    """A gated feed-forward whose gate is cut at ``limit`` from above and whose other branch is
    cut on both sides and shifted by one."""
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(logits, correction, router, margins=None):
    """Weights [T, experts]. ``margins``: a list that receives, per token, by how much (in choice
    scores relative to the last chosen score) the choice was made."""
    T, E = logits.shape
    s = torch.softmax(logits, -1)
    out = torch.zeros_like(s)
    margin = torch.full((T,), math.inf, dtype=torch.float64)
    for t in range(T):
        choice = s[t] + correction
        ranked = sorted(range(E), key=lambda e: (-float(choice[e]), e))
        chosen = ranked[:router["top"]]
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            out[t, e] = s[t, e] / total * router["scale"]
        if router["top"] < E:
            margin[t] = float(choice[chosen[-1]] - choice[ranked[router["top"]]])
    if margins is not None:
        margins.append(margin)
    return out


def experts(h, w, m, p, margins=None):
    weights = route(h @ w[p + "router"].T, w[p + "correction"], m["router"], margins)
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        out = out + weights[:, e:e + 1] * clamped_unit(h, w, m["expert"]["limit"], f"{p}e{e}.")
    if m.get("shared"):
        out = out + clamped_unit(h, w, m["shared"]["limit"], p + "shared.")
    return out


FEED_FORWARDS = {"dense": dense, "moe": experts}


# --------------------------------------------------------------------------- the model


def forward(config, weights, tokens, kind=torch.float64, states=None, margins=None):
    """Logits [T, vocab] of one sequence. ``states``: a list that receives the stream after every
    layer; ``margins``: see ``route``."""
    w = {name: t.to(kind) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    norm = lambda x, name: layer_norm(x, w[name], w[name + ".b"], eps)
    rule = (config.get("embedding") or {}).get("bigram")
    x = embedding(w, rule, tokens) if rule else w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    shared = {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](norm(x, p + "norm1"), w, layer["mixer"], eps, p + "mix.", shared)
        x = x + norm(y, p + "norm1b")
        if layer.get("mlp") is not None:
            y = FEED_FORWARDS[layer["mlp"]["kind"]](norm(x, p + "norm2"), w, layer["mlp"], p + "mlp.",
                                                    margins)
            x = x + norm(y, p + "norm2b")
        if states is not None:
            states.append(x)
    return norm(x, "final.norm") @ w["head"].T


def load(model_dir):
    path = Path(model_dir)
    return json.loads((path / "config.json").read_text()), read_tensors(path / "model.safetensors")

"""Tiny Susalorn configurations for the tests, with weights drawn large enough that every
mechanism moves the logits.

The configurations differ in every size: width, vocabulary, the number of streams (1 to 5),
latent attention (one to six heads; unrotated dimensions shorter and longer than the rotated
part, rotated parts that turn in whole or in part; latents that are multiples of 32, of 16, of
neither; values longer and shorter than keys; with and without scaled frequencies), the delta
rule (value heads that share a key head, one to six; keys from 8 to 130 values; values that fit
the single-token kernel and values that do not; one tap to six; inner sizes that are and are not
multiples of 8), feed-forwards (gated, absent, routed: with groups of which some or all are kept,
without groups, one expert of many, all of them), and the order of the layers (no loop, a loop
from the start, in the middle, over one layer).
"""

from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mlp, base=10000.0, scaling=None,
           dims=None):
    rot = {"base": base, "dims": dims or rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "scale": scale,
                      "kv_rank": kv_rank, "q_rank": q_rank, "rot": rot}}


def delta(heads, kv_heads, dim, vdim, conv, mlp, ranks=(8, 16)):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                      "decay_rank": ranks[0], "gate_rank": ranks[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


YARN = (8.0, 64, 16.0, 0.5)

# four streams, a loop over the first two layers, rows of 48 + 16 = 64, pairs of value heads on a
# key head, three groups of three experts of which one is kept
S1 = {"architecture": "Susalorn", "vocab": 300, "width": 64, "norm": {"eps": 1e-5}, "streams": 4,
      "layers": [latent(4, 24, 16, 32, 48, 40, 0.2, moe(9, 2, 40, (3, 1), 1.5), scaling=YARN),
                 delta(4, 2, 16, 24, 3, dense(96)),
                 latent(4, 24, 16, 32, 48, 40, 0.2, None, scaling=YARN)],
      "loop": {"start": 0, "stop": 2, "times": 2}}

# two streams, no experts, no loop, nothing a multiple of 8: a row of 40 + 6 values, queries' latent
# of 22, inner sizes of 5 and 7, one tap (no inputs kept), three value heads on one key head
S2 = {"architecture": "Susalorn", "vocab": 257, "width": 96, "norm": {"eps": 1e-6}, "streams": 2,
      "layers": [delta(3, 1, 20, 10, 1, dense(64), (5, 7)),
                 latent(3, 4, 6, 20, 40, 22, 0.4, dense(100), base=500.0),
                 delta(3, 3, 9, 14, 2, None, (3, 12))]}

# one stream, one head of everything, six taps, one expert of five, a loop over one layer
S3 = {"architecture": "Susalorn", "vocab": 64, "width": 36, "norm": {"eps": 1e-5}, "streams": 1,
      "layers": [latent(1, 8, 2, 12, 16, 8, 0.5, moe(5, 1, 24), base=100.0, scaling=(2.0, 16, 4.0, 1.0)),
                 delta(1, 1, 8, 16, 6, moe(3, 3, 16, None, 0.7))],
      "loop": {"start": 1, "stop": 2, "times": 3}}

# five streams, no experts, rows of 128 + 32, keys of 128 in heads that keep 16-bit rows in
# registers, a rotated part that turns in half, a loop in the middle
S4 = {"architecture": "Susalorn", "vocab": 512, "width": 128, "norm": {"eps": 2e-6}, "streams": 5,
      "layers": [delta(2, 1, 128, 64, 4, dense(192), (32, 64)),
                 latent(5, 32, 32, 16, 128, 64, 0.15, dense(192), base=1000000.0, dims=16,
                        scaling=(4.0, 256, 32.0, 1.0)),
                 delta(4, 4, 48, 32, 4, None, (24, 128)),
                 latent(2, 64, 32, 80, 128, 48, 0.12, dense(96))],
      "loop": {"start": 1, "stop": 3, "times": 2}}

# three streams, values of 136 (no single-token kernel), keys of 130, all groups kept, experts
# whose width is no multiple of 8
S5 = {"architecture": "Susalorn", "vocab": 100, "width": 72, "norm": {"eps": 3e-6}, "streams": 3,
      "layers": [delta(2, 2, 40, 136, 4, moe(6, 4, 20, (3, 3), 2.5)),
                 latent(2, 10, 4, 24, 18, 12, 0.35, moe(16, 3, 12, (2, 1)), base=50.0),
                 delta(1, 1, 130, 24, 5, moe(4, 2, 48, (4, 2), 0.5))]}

CONFIGS = {"S1": (S1, 41, 16), "S2": (S2, 42, 8), "S3": (S3, 43, 4), "S4": (S4, 44, 16),
           "S5": (S5, 45, 2)}   # config, seed, page


def draw_tensors(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Weights for ``config``, by the names and shapes of the engine's weight contract: matrices
    ~ N(0, 1/in) (the embedding N(0, 1), routers three times as wide so that scores differ),
    norm weights around 1, convolutions ~ N(0, 0.5); streams are read with weights around 1 / n and
    mixed by the identity + N(0, 0.1), and every sublayer's output enters with about 0.7; A_log
    around -2 and dt_bias around -1, so that a state keeps what it saw for tens of tokens, some
    channels far longer than others; sinks around 1."""
    from mlx_one_b200.architectures.susalorn import describe
    from mlx_one_b200.config.susalorn import SusalornConfig
    from mlx_one_b200.parts import expected_tensors

    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, want in expected_tensors(describe(SusalornConfig.from_dict(config))).items():
        values = torch.randn(want.shape, generator=generator)
        if name.endswith(".A_log"):
            values = -2.0 + 0.7 * values
        elif name.endswith(".dt_bias"):
            values = -1.0 + 1.0 * values
        elif name.endswith(".sink"):
            values = 1.0 + values
        elif name.endswith(".in"):
            values = (1.0 + 0.5 * values) / want.shape[0]
        elif name.endswith(".out"):
            values = 0.7 + 0.2 * values
        elif want.init == "mix":
            values = torch.eye(want.shape[0]) + 0.1 * values
        elif want.init == "norm":
            values = 1.0 + 0.2 * values
        elif name.endswith(".router"):
            values = 3.0 * values / want.shape[1] ** 0.5
        elif name == "embed":
            pass
        elif name.endswith(".conv"):
            values = 0.5 * values
        elif len(want.shape) == 2:
            values = values / want.shape[1] ** 0.5
        else:
            values = 0.3 * values
        out[name] = values.to(torch.bfloat16)
    return out


def write_model(folder: Path, config: dict, seed: int) -> Path:
    """The folder of a model: its config.json as a user would write it, without the inner sizes
    that the stored tensors decide."""
    from mlx_one_b200.weights.safetensors_io import write_safetensors

    write_safetensors(folder / "model.safetensors", draw_tensors(config, seed), {"format": "pt"})
    bare = json.loads(json.dumps(config))
    for layer in bare["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"].pop(key, None)
    (folder / "config.json").write_text(json.dumps(bare, indent=1))
    return folder


def make_model_dir(name: str, root: Path | None = None, config: dict | None = None) -> Path:
    """Writes the tiny model ``name`` into a fresh temporary folder (never into the repo)."""
    base, seed, _ = CONFIGS[name]
    folder = Path(tempfile.mkdtemp(prefix=f"tiny_{name}_", dir=root))
    return write_model(folder, base if config is None else config, seed)


class PlainModel:
    """The plain implementation on a model folder: logits of whole sequences in 64-bit."""

    def __init__(self, folder):
        import plain_susalorn

        self.plain = plain_susalorn
        self.config, self.weights = plain_susalorn.load(folder)

    def logits(self, tokens, streams=None):
        """float32 [T, vocab] with ``margin`` [T]: by how much, in router logits, the position's
        closest choice of experts was made (infinite without routed layers)."""
        margins = []
        out = self.plain.forward(self.config, self.weights, list(tokens), streams=streams,
                                 margins=margins).float()
        out.margin = torch.stack(margins).amin(0).float() if margins \
            else torch.full((out.shape[0],), float("inf"))
        return out

    def greedy(self, prompt, count):
        tokens, out = list(prompt), []
        for _ in range(count):
            out.append(int(self.logits(tokens)[-1].argmax()))
            tokens.append(out[-1])
        return out


# bfloat16: a row's error is the root mean square over the vocabulary of (engine - plain), its
# mean taken off, relative to the spread of the plain logits. Rounding alone gives a few percent
# on these models; a wrong key, a lost state or a token fed twice gives 15 % and more.
BF16_ROW_ERROR = 0.12
# The bfloat16 engine routes what its own 16-bit arithmetic has made of the streams, so a position
# whose routing margin is below this may go to other experts than in the plain model; its logits
# are then others, and so, a little, are those of every later position of the request. Rows from
# the first such position on are not compared in bfloat16; the 32-bit engine is compared
# everywhere, and so is bfloat16 on models without routed experts.
ROUTING_MARGIN = 0.1


def assert_rows_close(got, want, dtype, what: str = "") -> None:
    """float32: every logit within 3e-4 + 3e-4 |plain| (positions with a routing margin below 1e-4
    left out, and those behind them). bfloat16: every row's error (see above) within
    ``BF16_ROW_ERROR`` up to the request's first position that is routed by a hair."""
    margin = getattr(want, "margin", None)
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    margin = torch.full((want.shape[0],), float("inf")) if margin is None else margin.float().cpu()
    hair = 1e-4 if dtype == torch.float32 else ROUTING_MARGIN
    settled = torch.cumsum((margin < hair).float(), 0) == 0
    if dtype == torch.float32:
        excess = (got - want).abs() - (3e-4 + 3e-4 * want.abs())
        excess[~settled] = -1
        assert excess.max() <= 0, (f"{what}: logits differ by {(got - want).abs().max():.3e}; rows "
                                   f"{torch.nonzero((excess > 0).any(-1)).flatten().tolist()[:8]}")
        return
    difference = got - want
    difference = difference - difference.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    rows = difference.pow(2).mean(-1).sqrt() / spread
    assert torch.isfinite(rows).all(), f"{what}: logits that are not finite"
    bad = (rows > BF16_ROW_ERROR) & settled
    assert not bad.any(), (f"{what}: row error {rows[settled].max():.3f} of the spread; rows "
                           f"{torch.nonzero(bad).flatten().tolist()[:8]}")

"""Tiny Zinizen configurations for the tests, with weights drawn large enough that every
mechanism moves the logits.

The configurations differ in every size: width, vocabulary, the second table's buckets (none at
all in one), attention (one to six query heads on one to three key heads, queries and keys of 8 to
128 values, values longer, shorter and of the same size, head counts that are no power of two;
capped and uncapped scores, with and without a temperature, values mixed in some layers and not
in others), latent attention (one to five heads, values longer and shorter than keys, rotated
parts that turn in whole or in part), the recurrence (as wide as the model and not; parts of 64, 8,
5 and of 1 channel; one tap to six), feed-forwards (dense, absent, routed: one expert of many, all
of them, with and without a shared one whose limit is its own), and the order of the layers.
"""

from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, scale, mlp, softcap=None, temp=None, mix=False):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        mixer["softcap"] = softcap
    if temp is not None:
        mixer["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if mix:
        mixer["v_mix"] = True
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mlp, base=10000.0, dims=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "scale": scale,
                      "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": dims or rot_dim}}}


def rglru(width, blocks, conv, mlp):
    return {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, scale=1.0, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
           "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def bigram(buckets, mul_prev, mul_cur):
    return {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}


# every mixer and feed-forward; pairs of query heads on a key head, values shorter than keys
Z1 = {"architecture": "Zinizen", "vocab": 300, "width": 64, "norm": {"eps": 1e-5},
      "embedding": bigram(101, 7, 13),
      "layers": [attention(4, 2, 32, 16, 0.25, dense(96), 8.0, (0.4, 16), True),
                 rglru(96, 3, 3, moe(9, 2, 40, 0.8, 1.5, (48, 1.2))),
                 latent(3, 24, 8, 32, 48, 40, 0.2, moe(6, 3, 24, 1.0, 1.0, (16, 0.5))),
                 attention(2, 1, 24, 32, 0.3, None, 5.0, (0.2, 24), True),
                 attention(4, 2, 32, 16, 0.25, dense(64), 8.0, (0.4, 16), True)]}

# nothing a multiple of 8: three query heads on one key head of 20 values, values of 28, scores
# without a cap, no temperature, parts of five channels, one tap, experts without a shared one
Z2 = {"architecture": "Zinizen", "vocab": 257, "width": 52, "norm": {"eps": 1e-6},
      "embedding": bigram(11, 3, 1),
      "layers": [rglru(35, 7, 1, dense(50)),
                 attention(3, 1, 20, 28, 0.3, moe(5, 1, 20, 1.5, 2.5)),
                 latent(2, 6, 4, 10, 18, 22, 0.4, None, base=500.0, dims=2),
                 attention(3, 3, 18, 14, 0.35, dense(30), None, (0.5, 7), True),
                 attention(6, 3, 10, 14, 0.4, None, 3.0, None, True)]}

# one head, one key head, one part, one expert, six taps, no second table; keys and values of
# equal size
Z3 = {"architecture": "Zinizen", "vocab": 64, "width": 36, "norm": {"eps": 1e-5},
      "layers": [attention(1, 1, 16, 16, 0.4, moe(1, 1, 16, 0.7, 1.0, (8, 2.0)), 50.0, (0.3, 1), True),
                 rglru(8, 1, 6, moe(4, 4, 24, 0.9, 0.7)),
                 latent(1, 8, 2, 12, 16, 8, 0.5, dense(40), base=100.0)]}

# rows of 64 values (prompts on the tcgen05 kernel), four query heads on a key head, parts of 64
# channels, one value mixer that no later layer follows
Z4 = {"architecture": "Zinizen", "vocab": 512, "width": 128, "norm": {"eps": 2e-6},
      "embedding": bigram(1000, 29, 11),
      "layers": [rglru(192, 3, 4, dense(192)),
                 attention(8, 2, 64, 48, 0.125, moe(8, 2, 64, 1.1, 2.0, (64, 0.6)), 30.0, (0.3, 32), True),
                 latent(5, 32, 32, 48, 128, 64, 0.15, dense(200), base=1000000.0),
                 attention(4, 4, 48, 64, 0.15, dense(96), 20.0),
                 rglru(64, 8, 2, None)]}

# heads of 128 values, head counts that are no power of two, parts of one channel
Z5 = {"architecture": "Zinizen", "vocab": 100, "width": 72, "norm": {"eps": 3e-6},
      "embedding": bigram(5, 2, 3),
      "layers": [attention(6, 2, 128, 128, 0.1, moe(6, 4, 20, 1.0, 2.5, (36, 1.0)), 12.0, (0.25, 50), False),
                 attention(5, 5, 112, 40, 0.12, dense(64), 9.0, (0.25, 3), True),
                 rglru(24, 24, 5, moe(16, 3, 12, 1.3, 1.0, (10, 0.9))),
                 attention(10, 5, 16, 40, 0.3, dense(72), 40.0, None, True)]}

CONFIGS = {"Z1": (Z1, 51, 16), "Z2": (Z2, 52, 8), "Z3": (Z3, 53, 4), "Z4": (Z4, 54, 16),
           "Z5": (Z5, 55, 2)}   # config, seed, page


def draw_tensors(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Weights for ``config``, by the names and shapes of the engine's weight contract: matrices
    ~ N(0, 1/in) (tables N(0, 1), routers three times as wide so that scores differ), norm weights
    around 1 and their biases ~ N(0, 0.3), convolutions ~ N(0, 0.5), lam around -3.5 so that a
    state keeps what it saw for tens of tokens, some channels far longer than others, corrections
    of the size of a score, mixing factors around 0.5."""
    from mlx_one_b200.architectures.zinizen import describe
    from mlx_one_b200.config.zinizen import ZinizenConfig
    from mlx_one_b200.parts import expected_tensors

    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, want in expected_tensors(describe(ZinizenConfig.from_dict(config))).items():
        values = torch.randn(want.shape, generator=generator)
        if name.endswith(".lam"):
            values = -3.5 + 1.5 * values
        elif name.endswith(".vmix"):
            values = 0.5 + 0.2 * values
        elif name.endswith(".correction"):
            values = 0.1 * values
        elif want.init == "norm":
            values = 1.0 + 0.2 * values
        elif name.endswith(".router"):
            values = 3.0 * values / want.shape[1] ** 0.5
        elif name in ("embed", "bigram"):
            pass
        elif name.endswith(".conv"):
            values = 0.5 * values
        elif name.endswith((".ra", ".ri")):
            values = 1.5 * values / want.shape[2] ** 0.5
        elif len(want.shape) == 2:
            values = (2.0 if name.endswith((".gate", ".up")) else 1.0) * values / want.shape[1] ** 0.5
        else:
            values = 0.3 * values
        out[name] = values.to(torch.bfloat16)
    return out


def write_model(folder: Path, config: dict, seed: int) -> Path:
    from mlx_one_b200.weights.safetensors_io import write_safetensors

    write_safetensors(folder / "model.safetensors", draw_tensors(config, seed), {"format": "pt"})
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    return folder


def make_model_dir(name: str, root: Path | None = None, config: dict | None = None) -> Path:
    """Writes the tiny model ``name`` into a fresh temporary folder (never into the repo)."""
    base, seed, _ = CONFIGS[name]
    folder = Path(tempfile.mkdtemp(prefix=f"tiny_{name}_", dir=root))
    return write_model(folder, base if config is None else config, seed)


class PlainModel:
    """The plain implementation on a model folder: logits of whole sequences in 64-bit."""

    def __init__(self, folder):
        import plain_zinizen

        self.plain = plain_zinizen
        self.config, self.weights = plain_zinizen.load(folder)

    def logits(self, tokens, states=None):
        """float32 [T, vocab] with ``margin`` [T]: by how much, in choice scores, the position's
        closest choice of experts was made (infinite without routed layers)."""
        margins = []
        out = self.plain.forward(self.config, self.weights, list(tokens), states=states,
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
# The bfloat16 engine routes what its own 16-bit arithmetic has made of the stream, so a position
# whose routing margin is below this may go to other experts than in the plain model; its logits
# are then others, and so, a little, are those of every later position of the request. Rows from
# the first such position on are not compared in bfloat16; the 32-bit engine is compared
# everywhere, and so is bfloat16 on models without routed experts.
ROUTING_MARGIN = 0.015


def assert_rows_close(got, want, dtype, what: str = "") -> None:
    """float32: every logit within 4e-4 + 4e-4 |plain| (positions with a routing margin below 2e-5
    left out, and those behind them). bfloat16: every row's error (see above) within
    ``BF16_ROW_ERROR`` up to the request's first position that is routed by a hair."""
    margin = getattr(want, "margin", None)
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    margin = torch.full((want.shape[0],), float("inf")) if margin is None else margin.float().cpu()
    hair = 2e-5 if dtype == torch.float32 else ROUTING_MARGIN
    settled = torch.cumsum((margin < hair).float(), 0) == 0
    if dtype == torch.float32:
        excess = (got - want).abs() - (4e-4 + 4e-4 * want.abs())
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

"""Zinizen models whose every size and constant is drawn at random (seeded): the 32-bit and the
bfloat16 engine against the plain model over whole requests, decoded tails, portions and mixed
batches."""

import random

import pytest
import torch

from test_gpu_susalorn import engine
from tiny_models import cut, mixed_schedule, prompts, replay
from zinizen_models import (PlainModel, assert_rows_close, attention, bigram, dense, latent, moe, rglru,
                            write_model)

pytestmark = pytest.mark.gpu


def random_config(seed: int) -> dict:
    rng = random.Random(seed)
    width = rng.choice([40, 48, 52, 64, 80, 96, 128, 160, 192, 264])

    def feed_forward():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < (0.9 if seed % 2 else 0.5):         # every second model is mostly dense
            return dense(rng.choice([32, 40, 96, 200, 256]))
        experts = rng.choice([1, 2, 3, 5, 8, 12, 24])
        shared = None if rng.random() < 0.4 else (rng.choice([8, 20, 48, 64]), rng.uniform(0.4, 3.0))
        return moe(experts, rng.randint(1, min(5, experts)), rng.choice([16, 20, 24, 36, 64]),
                   rng.uniform(0.4, 3.0), rng.choice([0.5, 1.0, 2.5]), shared)

    # the values of every layer that mixes them have the same size in all
    kv, vdim = rng.choice([(1, 16), (1, 64), (2, 8), (2, 24), (2, 64), (3, 10), (4, 32), (2, 128)])

    def attention_layer():
        mix = rng.random() < 0.7
        kv_heads, values = (kv, vdim) if mix else (rng.choice([1, 2, 3, 4]), rng.choice([8, 20, 32, 64, 96]))
        dim = rng.choice([8, 12, 16, 32, 48, 64, 64, 80, 128])
        return attention(kv_heads * rng.choice([1, 2, 3, 4]), kv_heads, dim, values, rng.uniform(0.5, 2.0) / dim ** 0.5,
                         feed_forward(), None if rng.random() < 0.2 else rng.choice([1.5, 5.0, 20.0, 50.0]),
                         None if rng.random() < 0.2 else (rng.uniform(-0.2, 0.6), rng.choice([1, 5, 16, 50, 100])), mix)

    def latent_layer():
        rot_dim = rng.choice([2, 4, 8, 16, 24, 32, 64])
        return latent(rng.choice([1, 2, 3, 4, 6, 8, 12, 17]), rng.choice([4, 8, 16, 24, 32, 48, 64, 96]),
                      rot_dim, rng.choice([8, 16, 20, 32, 64, 96]), rng.choice([8, 16, 24, 40, 64, 96, 128, 192]),
                      rng.choice([8, 12, 24, 40, 64, 100]), rng.uniform(0.05, 0.3), feed_forward(),
                      base=rng.choice([100.0, 10000.0, 1000000.0]))

    def recurrent_layer():
        blocks = rng.choice([1, 2, 3, 4, 8])
        return rglru(blocks * rng.choice([1, 5, 8, 16, 24, 64, 72]), blocks, rng.choice([1, 2, 3, 4, 4, 5]), feed_forward())

    count = rng.randint(3, 7)
    kinds = [rng.choice("alr") for _ in range(count)]
    for place, kind in zip(rng.sample(range(count), 3), "alr"):
        kinds[place] = kind
    make = {"a": attention_layer, "l": latent_layer, "r": recurrent_layer}
    config = {"architecture": "Zinizen", "vocab": rng.randint(50, 700), "width": width,
              "norm": {"eps": rng.choice([1e-6, 1e-5])}, "layers": [make[kind]() for kind in kinds]}
    if rng.random() < 0.85:
        config["embedding"] = bigram(rng.choice([1, 7, 100, 997]), rng.randint(0, 1000), rng.randint(1, 99999))
    return config


@pytest.mark.parametrize("seed", range(16))
def test_a_model_drawn_at_random(tmp_path, seed):
    config = random_config(seed)
    write_model(tmp_path, config, 100 + seed)
    plain = PlainModel(tmp_path)
    page = (16, 16, 8, 4, 32, 64)[seed % 6]
    lengths = (150, 64, 23, 50, 9, 2, 1)
    requests = dict(enumerate(prompts(config["vocab"], lengths, seed=seed)))
    want = {key: plain.logits(tokens) for key, tokens in requests.items()}
    for dtype in (torch.float32, torch.bfloat16):
        runner, cache = engine(tmp_path, dtype, page, 4 * 192, max_requests=4)
        tokens = requests[0]
        got = replay(runner, cache, [([("w", tokens)], ["w"])])["w"]
        assert_rows_close(got, want[0], dtype, f"seed {seed} whole")
        steps = [([("d", tokens[:110])], [])] + [([("d", [t])], []) for t in tokens[110:]]
        steps[-1] = (steps[-1][0], ["d"])
        assert_rows_close(replay(runner, cache, steps)["d"], want[0], dtype, f"seed {seed} decoded tail")
        steps = [([("p", part)], []) for part in cut(tokens, (7, 2, 40, 3, 1))]
        steps[-1] = (steps[-1][0], ["p"])
        assert_rows_close(replay(runner, cache, steps)["p"], want[0], dtype, f"seed {seed} portions")
        got = replay(runner, cache, mixed_schedule(requests))
        for key in requests:
            assert_rows_close(got[key], want[key], dtype, f"seed {seed} mixed request {key}")
        assert not cache.requests()

"""Susalorn models whose every size and constant is drawn at random (seeded): the 32-bit and the
bfloat16 engine against the plain model over whole requests, decoded tails, portions and mixed
batches."""

import random

import pytest
import torch

from susalorn_models import PlainModel, assert_rows_close, delta, dense, latent, moe, write_model
from tiny_models import cut, mixed_schedule, prompts, replay

pytestmark = pytest.mark.gpu
DEVICE = "cuda:0"


def random_config(seed: int) -> dict:
    rng = random.Random(seed)
    width = rng.choice([40, 48, 64, 80, 96, 128, 160, 192, 264])

    def feed_forward():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < (0.9 if seed % 2 else 0.5):         # every second model is mostly dense
            return dense(rng.choice([32, 40, 96, 200, 256]))
        groups = rng.choice([None, 2, 3, 4])
        per = rng.choice([1, 2, 3, 4, 8])
        keep = rng.randint(1, groups) if groups else 1
        experts = per * (groups or 1)
        return moe(experts, rng.randint(1, min(4, per * keep)), rng.choice([16, 24, 36, 64]),
                   (groups, keep) if groups else None, rng.choice([0.5, 1.0, 2.5]))

    def latent_layer():
        rot_dim = rng.choice([2, 4, 8, 16, 24, 32, 64])
        scaling = None if rng.random() < 0.3 else (rng.choice([1.0, 2.0, 8.0, 32.0]), rng.choice([16, 64, 512, 4096]),
                                                   rng.choice([4.0, 16.0, 32.0]), rng.choice([0.5, 1.0, 2.0]))
        return latent(rng.choice([1, 2, 3, 4, 6, 8, 12, 17]), rng.choice([4, 8, 16, 24, 32, 48, 64, 96]),
                      rot_dim, rng.choice([8, 16, 20, 32, 64, 96]),
                      rng.choice([8, 16, 24, 40, 64, 96, 128, 160, 192]), rng.choice([8, 12, 24, 40, 64, 100]),
                      rng.uniform(0.05, 0.3), feed_forward(), base=rng.choice([100.0, 10000.0, 1000000.0]),
                      scaling=scaling)

    def delta_layer():
        kv_heads = rng.choice([1, 2, 3, 4])
        return delta(kv_heads * rng.choice([1, 2, 3]), kv_heads, rng.choice([8, 12, 16, 24, 32, 48, 64, 100, 128]),
                     rng.choice([8, 10, 16, 24, 32, 64, 128, 132]), rng.choice([1, 2, 3, 4, 4, 4, 5]), feed_forward(),
                     (rng.choice([3, 8, 16, 24, 64]), rng.choice([4, 8, 10, 32, 132])))

    count = rng.randint(2, 6)
    kinds = [rng.choice("ld") for _ in range(count)]
    kinds[rng.randrange(count)] = "l"
    kinds[(kinds.index("l") + 1) % count] = "d"
    config = {"architecture": "Susalorn", "vocab": rng.randint(50, 700), "width": width,
              "norm": {"eps": rng.choice([1e-6, 1e-5])}, "streams": rng.choice([1, 2, 3, 4, 4, 6, 9]),
              "layers": [latent_layer() if kind == "l" else delta_layer() for kind in kinds]}
    if rng.random() < 0.6:
        start = rng.randrange(count)
        config["loop"] = {"start": start, "stop": rng.randint(start + 1, count), "times": rng.randint(1, 3)}
    return config


def engine(folder, dtype, page_size, capacity, max_requests=4):
    from mlx_one_b200.cache import CacheManager
    from mlx_one_b200.engine.loading import load_model
    from mlx_one_b200.engine.runner import Runner

    loaded = load_model(folder, dtype, DEVICE)
    cache = CacheManager(loaded.model.cache_needs, page_size=page_size, capacity_tokens=capacity,
                         max_requests=max_requests, dtype=dtype, device=DEVICE)
    return Runner(loaded.model, cache), cache


@pytest.mark.parametrize("seed", range(14))
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

"""Zinizen without a GPU: configuration, weight names, what the cache keeps, the plain mechanisms
themselves, and the engine's bookkeeping (normed updates, pages of two kinds, state slots, the
second table's last token, values left for later layers) run with the plain kernel set against the
plain model."""

import copy
import json
import math

import pytest
import torch

import plain_zinizen as plain
from plain_ops import PlainOps
from tiny_models import cut, mixed_schedule, prompts, replay
from zinizen_models import CONFIGS, Z1, Z2, Z3, PlainModel, assert_rows_close, make_model_dir


def engine(folder, page_size, capacity, max_requests=4):
    from mlx_one_b200.cache import CacheManager
    from mlx_one_b200.engine.loading import load_model
    from mlx_one_b200.engine.runner import Runner

    loaded = load_model(folder, "float32", "cpu", PlainOps())
    cache = CacheManager(loaded.model.cache_needs, page_size=page_size, capacity_tokens=capacity,
                         max_requests=max_requests, dtype=torch.float32, device="cpu")
    return Runner(loaded.model, cache), cache


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zinizen_cpu")
    return {name: make_model_dir(name, root) for name in CONFIGS}


# ------------------------------------------------------------------ configuration


def test_config_round_trip_and_registry(tmp_path):
    from mlx_one_b200.config import ZinizenConfig, read_config

    for name, (config, _, _) in CONFIGS.items():
        typed = ZinizenConfig.from_dict(config)
        assert ZinizenConfig.from_dict(typed.to_dict()) == typed, name
    (tmp_path / "config.json").write_text(json.dumps(Z1))
    entry, typed = read_config(tmp_path)
    assert entry.name == "zinizen" and typed.width == 64 and typed.bigram.buckets == 101
    first = typed.layers[0].mixer
    assert first.softcap == 8.0 and first.q_temp.every == 16.0 and first.v_mix
    assert typed.layers[1].mixer.blocks == 3 and typed.layers[1].mlp.shared.limit == 1.2
    assert typed.layers[3].mlp is None and typed.first_mixed == 0
    second = ZinizenConfig.from_dict(Z2)
    assert second.layers[1].mixer.softcap is None and second.layers[1].mixer.q_temp is None
    assert second.layers[1].mlp.shared is None and second.first_mixed == 3
    assert ZinizenConfig.from_dict(Z3).bigram is None


@pytest.mark.parametrize("path, value, text", [
    (("layers", 0, "type"), "mamba2", "type"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "softcap"), 0, "softcap"),
    (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
    (("layers", 0, "mixer", "v_mix"), 1, "v_mix"),
    (("layers", 3, "mixer", "vdim"), 30, "mixed"),
    (("layers", 1, "mixer", "blocks"), 5, "blocks"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 2, "mixer", "rot", "dims"), 7, "dims"),
    (("layers", 2, "mixer", "rot", "dims"), 64, "dims"),
    (("layers", 1, "mlp", "kind"), "gated", "kind"),
    (("layers", 1, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 1, "mlp", "router", "top"), 10, "top"),
    (("embedding", "bigram", "buckets"), 0, "buckets"),
    (("embedding", "bigram", "mul_prev"), -1, "mul_prev"),
    (("norm", "eps"), -1.0, "eps"),
])
def test_config_rejections(path, value, text):
    from mlx_one_b200.config import ConfigError, ZinizenConfig

    config = copy.deepcopy(Z1)
    at = config
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=text):
        ZinizenConfig.from_dict(config)


def test_missing_key_is_named():
    from mlx_one_b200.config import ConfigError, ZinizenConfig

    for path, text in ((("layers", 0, "mixer", "scale"), r"layers\[0\]\.mixer\.scale"),
                       (("layers", 0, "mixer", "q_temp", "coef"), r"layers\[0\]\.mixer\.q_temp\.coef"),
                       (("layers", 1, "mixer", "width"), r"layers\[1\]\.mixer\.width"),
                       (("layers", 1, "mlp", "shared", "limit"), r"layers\[1\]\.mlp\.shared\.limit"),
                       (("layers", 2, "mixer", "q_rank"), r"layers\[2\]\.mixer\.q_rank"),
                       (("width",), "width")):
        config = copy.deepcopy(Z1)
        at = config
        for key in path[:-1]:
            at = at[key]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=text):
            ZinizenConfig.from_dict(config)


def test_weight_names_and_what_the_cache_keeps():
    from mlx_one_b200.architectures.zinizen import describe
    from mlx_one_b200.config import ZinizenConfig
    from mlx_one_b200.parts import FixedState, PagedKeyValues, cache_entries, expected_tensors

    spec = describe(ZinizenConfig.from_dict(Z1))
    shapes = {name: tuple(want.shape) for name, want in expected_tensors(spec).items()}
    assert shapes["embed"] == (300, 64) and shapes["bigram"] == (102, 64) and shapes["head"] == (300, 64)
    assert shapes["l0.mix.q"] == (128, 64) and shapes["l0.mix.v"] == (32, 64)
    assert shapes["l0.mix.q.norm"] == (128,) and shapes["l0.mix.k.norm"] == (64,)
    assert shapes["l0.mix.vmix"] == () and shapes["l0.mix.o"] == (64, 64)
    assert shapes["l1.mix.ra"] == (3, 32, 32) and shapes["l1.mix.ri.b"] == (3, 32)
    assert shapes["l1.mix.conv"] == (96, 3) and shapes["l1.mix.lam"] == (96,)
    assert shapes["l2.mix.g"] == (3, 64) and shapes["l2.mix.uv"] == (96, 48)
    assert shapes["l1.mlp.e8.gate"] == (40, 64) and shapes["l1.mlp.shared.up"] == (48, 64)
    assert shapes["l1.mlp.correction"] == (9,) and shapes["l0.mlp.up"] == (96, 64)
    assert shapes["l3.norm1b.b"] == (64,) and "l3.norm2" not in shapes and "l3.norm2b" not in shapes
    assert shapes["final.norm.b"] == (64,)
    needs = cache_entries(spec)
    assert needs[0] == needs[4] == PagedKeyValues(2, 32) and needs[3] == PagedKeyValues(1, 32)
    assert needs[2] == PagedKeyValues(1, 56, planes=1)
    assert needs[(1, "state")] == FixedState((96,), "float32") and needs[(1, "inputs")] == FixedState((2, 96))
    assert needs[(-1, "embedding")] == FixedState((1,), "int32") and len(needs) == 7
    second = cache_entries(describe(ZinizenConfig.from_dict(Z2)))
    assert (0, "inputs") not in second                       # one tap keeps nothing
    bare = expected_tensors(describe(ZinizenConfig.from_dict(Z2)))
    assert "l1.mix.vmix" not in bare and "l3.mix.vmix" in bare and "l1.mlp.shared.up" not in bare
    assert "bigram" not in expected_tensors(describe(ZinizenConfig.from_dict(Z3)))


def test_wrong_tensors_are_named(folders, tmp_path):
    from mlx_one_b200.engine.loading import load_model
    from mlx_one_b200.weights import WeightError
    from mlx_one_b200.weights.safetensors_io import write_safetensors

    tensors = plain.read_tensors(folders["Z1"] / "model.safetensors")
    (tmp_path / "config.json").write_text(json.dumps(Z1))
    del tensors["l3.mix.vmix"]
    tensors["l1.mix.ra"] = tensors["l1.mix.ra"][:2]
    tensors["l3.norm2"] = torch.zeros(64, dtype=torch.bfloat16)
    write_safetensors(tmp_path / "model.safetensors", tensors, {"format": "pt"})
    with pytest.raises(WeightError) as caught:
        load_model(tmp_path, "float32", "cpu", PlainOps())
    text = str(caught.value)
    assert "l3.mix.vmix" in text and "l1.mix.ra" in text and "l3.norm2" in text


def test_random_weights_mode(tmp_path):
    from mlx_one_b200.weights import write_random_model

    folder = write_random_model(tmp_path / "drawn", Z1, 3)
    runner, cache = engine(folder, 16, 64)
    (tokens,) = prompts(300, (9,), seed=1)
    got = replay(runner, cache, [([("r", tokens)], ["r"])])["r"]
    assert_rows_close(got, PlainModel(folder).logits(tokens), torch.float32, "drawn weights")


# ------------------------------------------------------------------ the plain mechanisms


def test_plain_attention_by_hand():
    """Two keys with equal products: only the distance tells them apart. A cap comes before the
    distance is taken off, and slopes halve from head to head as their count says."""
    assert plain.slopes(2, torch.float64).tolist() == [2.0 ** -4, 2.0 ** -8]
    assert plain.slopes(3, torch.float64)[0].item() == pytest.approx(2.0 ** (-8 / 3))
    q = torch.ones(2, 1, 1, dtype=torch.float64)
    k = torch.full((2, 1, 1), 30.0, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    out = plain.biased_attention(q, k, v, 1.0, 4.0, torch.tensor([0.5], dtype=torch.float64))
    assert out[0, 0, 0] == 1.0
    assert out[1, 0, 0].item() == pytest.approx(1 / (1 + math.exp(0.5)))
    k[0] = 60.0                              # capped: no more than the other
    again = plain.biased_attention(q, k, v, 1.0, 4.0, torch.tensor([0.5], dtype=torch.float64))
    assert again[1, 0, 0].item() == pytest.approx(out[1, 0, 0].item(), abs=1e-5)
    warm = plain.temperature([0, 6, 7, 15, 16], {"coef": 0.5, "every": 8}, torch.float64)
    assert warm[:2].tolist() == [1.0, 1.0]
    assert warm[2] == warm[4 - 1] - 0.5 * math.log(3) + 0.5 * math.log(2) == 1 + 0.5 * math.log(2)
    assert warm[4].item() == pytest.approx(1 + 0.5 * math.log(3))


def test_plain_recurrence_norms_routing_and_table_by_hand():
    one = lambda *values: torch.tensor([list(values)], dtype=torch.float64).T
    lam = torch.log(torch.expm1(torch.tensor([math.log(2) / 8], dtype=torch.float64)))   # a = 2^-r
    out = plain.linear_recurrence(one(2.0, 4.0), one(1.0, 1.0), one(1.0, 0.5), lam)
    root = math.sqrt(0.75)
    assert out[0].item() == pytest.approx(2 * root)          # the first token is no exception
    assert out[1].item() == pytest.approx(root + root * 2.0)
    u = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=torch.float64)
    m = torch.tensor([[[0.0, 1.0], [0.0, 0.0]], [[0.0, 0.0], [1.0, 0.0]]], dtype=torch.float64)
    assert plain.block_products(u, m, torch.zeros(2, 2)).tolist() == [[2.0, 0.0, 0.0, 3.0]]
    normed = plain.layer_norm(torch.tensor([1.0, 3.0]), torch.tensor([1.0, 2.0]), torch.tensor([0.0, 5.0]), 0.0)
    assert normed.tolist() == [-1.0, 7.0]
    # the correction chooses, the scores weigh
    logits = torch.log(torch.tensor([[0.5, 0.3, 0.2]], dtype=torch.float64))
    weights = plain.route(logits, torch.tensor([-1.0, 0.0, 0.0]), {"top": 2, "scale": 2.0})
    assert torch.allclose(weights, torch.tensor([[0.0, 1.2, 0.8]], dtype=torch.float64))
    table = {"embed": torch.zeros(5, 1), "bigram": torch.arange(8.0)[:, None]}
    rows = plain.embedding(table, {"buckets": 7, "mul_prev": 2, "mul_cur": 3}, [4, 1, 1])
    assert rows.flatten().tolist() == [7.0, (8 + 3) % 7, (2 + 3) % 7]
    # gate cut from above only, the other branch on both sides, shifted by one
    w = {"gate": torch.tensor([[9.0], [-9.0]]), "up": torch.tensor([[-9.0], [9.0]]), "down": torch.eye(2)}
    got = plain.clamped_unit(torch.ones(1, 1), w, 2.0, "")
    sigmoid = lambda z: 1 / (1 + math.exp(-z))
    assert got[0, 0].item() == pytest.approx(2 * sigmoid(3.404) * -1.0)
    assert got[0, 1].item() == pytest.approx(-9 * sigmoid(-9 * 1.702) * 3.0, rel=1e-4)


def test_every_mechanism_moves_the_logits(folders):
    model = PlainModel(folders["Z1"])
    (tokens,) = prompts(300, (60,), seed=2)
    want = model.logits(tokens)

    def moved(change):
        other = PlainModel(folders["Z1"])
        change(other)
        return float((other.logits(tokens) - want)[-10:].abs().max())

    def each(other, key, change):
        for layer in other.config["layers"]:
            if key in layer["mixer"]:
                change(layer["mixer"])

    def cap(other):
        each(other, "softcap", lambda m: m.pop("softcap"))

    def temperature(other):
        each(other, "q_temp", lambda m: m.pop("q_temp"))

    def mixing(other):
        other.config["layers"][4]["mixer"].pop("v_mix")

    def first(other):                     # the first layer that mixes is the first in order
        other.config["layers"][0]["mixer"].pop("v_mix")

    def second_table(other):
        other.config.pop("embedding")

    def limit(other):
        other.config["layers"][1]["mlp"]["expert"]["limit"] = 100.0

    def shared_limit(other):
        other.config["layers"][1]["mlp"]["shared"]["limit"] = 0.8

    def scale(other):
        other.config["layers"][1]["mlp"]["router"]["scale"] = 1.0

    def correction(other):
        other.weights["l1.mlp.correction"] = torch.zeros(9)

    def gate(other):
        other.weights["l2.mix.g"] = torch.zeros(3, 64)

    def bias(other):
        other.weights["l2.norm1b.b"] = torch.zeros(64)

    def decay(other):
        other.weights["l1.mix.lam"] = other.weights["l1.mix.lam"].float().mean().expand(96)

    for change in (cap, temperature, mixing, first, second_table, limit, shared_limit, scale, correction,
                   gate, bias, decay):
        assert moved(change) > 0.01, change.__name__


# ------------------------------------------------------------------ the engine's bookkeeping


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_portions_and_single_tokens(folders, name):
    config, _, page = CONFIGS[name]
    plain_model = PlainModel(folders[name])
    runner, cache = engine(folders[name], page, 256)
    (tokens,) = prompts(config["vocab"], (45,), seed=4)
    want = plain_model.logits(tokens)
    got = replay(runner, cache, [([("w", tokens)], ["w"])])["w"]
    assert_rows_close(got, want, torch.float32, f"{name} whole")
    for sizes in ((7, 2, 13, 1, 1, 3), (2,)):
        steps = [([("r", part)], []) for part in cut(tokens, sizes)]
        steps[-1] = (steps[-1][0], ["r"])
        assert_rows_close(replay(runner, cache, steps)["r"], want, torch.float32, f"{name} {sizes}")
    assert not cache.requests()


@pytest.mark.parametrize("name", ["Z1", "Z2"])
def test_the_stream_after_every_layer(folders, name):
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], page, 64)
    (tokens,) = prompts(config["vocab"], (19,), seed=2)
    seen = []

    def observe(place, residual, update):
        if place >= 0:
            seen.append(update.applied(residual))

    runner.model.observer = observe
    replay(runner, cache, [([("r", tokens)], ["r"])])
    runner.model.observer = None
    states = []
    PlainModel(folders[name]).logits(tokens, states)
    assert len(seen) == len(states) == len(config["layers"])
    for place, (got, want) in enumerate(zip(seen, states)):
        assert (got.double() - want).abs().max() < 2e-4, f"after layer {place}"


@pytest.mark.parametrize("name", ["Z1", "Z2", "Z5"])
def test_mixed_batches_with_pages_and_slots_used_again(folders, name):
    config, _, page = CONFIGS[name]
    plain_model = PlainModel(folders[name])
    lengths = (40, 30, 23, 17, 9, 2, 1)
    requests = dict(enumerate(prompts(config["vocab"], lengths, seed=5)))
    runner, cache = engine(folders[name], page, 3 * 64, max_requests=4)
    got = replay(runner, cache, mixed_schedule(requests))
    for request_id, tokens in requests.items():
        assert_rows_close(got[request_id], plain_model.logits(tokens), torch.float32,
                          f"{name} mixed request {request_id}")
    assert not cache.requests()
    cache.check()


def test_greedy_generation_through_the_entry_point(folders):
    """The engine's own entry point and scheduler: prompts in portions of eight tokens, three
    requests at a time, greedy tokens against the plain model's."""
    from mlx_one_b200 import BatchingConfig, CacheConfig, Engine, TextGenerationOptions

    config, _, page = CONFIGS["Z1"]
    plain_model = PlainModel(folders["Z1"])
    batch = prompts(config["vocab"], (7, 30, 3, 19), seed=8)
    engine_ = Engine(folders["Z1"], execution_dtype="float32", ops=PlainOps(), device="cpu",
                     cache_config=CacheConfig(block_size_tokens=page, capacity_tokens=256),
                     batching_config=BatchingConfig(max_sequences=3, prefill_chunk_size=8))
    results = engine_.generate_batch_ids(batch, TextGenerationOptions(max_tokens=6, ignore_eos=True))
    for prompt, result in zip(batch, results):
        assert list(result.token_ids) == plain_model.greedy(prompt, 6)
    engine_.close()

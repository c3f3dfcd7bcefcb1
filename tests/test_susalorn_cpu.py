"""Susalorn without a GPU: configuration, weight names and sizes that stored tensors decide, what
the cache keeps, the order of calls, the plain mechanisms themselves, and the engine's bookkeeping
(parallel streams, single-plane pages, state slots, a loop's passes) run with the plain kernel set
against the plain model."""

import copy
import json
import math

import pytest
import torch

import plain_susalorn as plain
from plain_ops import PlainOps
from susalorn_models import CONFIGS, S1, S2, S3, S4, PlainModel, assert_rows_close, make_model_dir
from tiny_models import cut, mixed_schedule, prompts, replay


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
    root = tmp_path_factory.mktemp("susalorn_cpu")
    return {name: make_model_dir(name, root) for name in CONFIGS}


# ------------------------------------------------------------------ configuration


def test_config_round_trip_and_registry(tmp_path):
    from mlx_one_b200.config import SusalornConfig, read_config

    for name, (config, _, _) in CONFIGS.items():
        typed = SusalornConfig.from_dict(config)
        assert SusalornConfig.from_dict(typed.to_dict()) == typed, name
    (tmp_path / "config.json").write_text(json.dumps(S1))
    entry, typed = read_config(tmp_path)
    assert entry.name == "susalorn" and typed.width == 64 and typed.streams == 4
    first = typed.layers[0]
    assert first.mixer.q_rank == 40 and first.mixer.rot.scaling.fast == 16.0
    assert first.mlp.groups == 3 and first.mlp.keep == 1 and first.mlp.scale == 1.5
    assert typed.layers[1].mixer.conv == 3 and typed.layers[2].mlp is None
    assert typed.loop.times == 2 and SusalornConfig.from_dict(S2).loop is None
    three = SusalornConfig.from_dict(S3)
    assert three.layers[0].mlp.groups == 1 and three.layers[0].mlp.scale == 1.0
    plain_rot = SusalornConfig.from_dict(S2).layers[1].mixer.rot
    assert plain_rot.scaling is None


@pytest.mark.parametrize("path, value, text", [
    (("layers", 0, "type"), "attention", "type"),
    (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "dims"),
    (("layers", 0, "mixer", "rot", "dims"), 64, "dims"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0, "factor"),
    (("layers", 0, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 0, "mlp", "kind"), "shared", "kind"),
    (("layers", 0, "mlp", "router", "groups", "count"), 4, "count"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5, "keep"),
    (("layers", 0, "mlp", "router", "top"), 5, "top"),
    (("loop", "stop"), 4, "loop"),
    (("streams",), 0, "streams"),
    (("norm", "eps"), -1.0, "eps"),
])
def test_config_rejections(path, value, text):
    from mlx_one_b200.config import ConfigError, SusalornConfig

    config = copy.deepcopy(S1)
    at = config
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=text):
        SusalornConfig.from_dict(config)


def test_missing_key_is_named():
    from mlx_one_b200.config import ConfigError, SusalornConfig

    for path, text in ((("layers", 0, "mixer", "rot", "base"), r"layers\[0\]\.mixer\.rot\.base"),
                       (("layers", 1, "mixer", "vdim"), r"layers\[1\]\.mixer\.vdim"),
                       (("layers", 0, "mlp", "router", "top"), r"layers\[0\]\.mlp\.router\.top"),
                       (("streams",), "streams")):
        config = copy.deepcopy(S1)
        at = config
        for key in path[:-1]:
            at = at[key]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=text):
            SusalornConfig.from_dict(config)


def test_order_of_calls_weight_names_and_what_the_cache_keeps():
    from mlx_one_b200.architectures.susalorn import describe
    from mlx_one_b200.config import SusalornConfig
    from mlx_one_b200.parts import FixedState, PagedKeyValues, cache_entries, expected_tensors

    spec = describe(SusalornConfig.from_dict(S1))
    assert [call.layer for call in spec.order] == [0, 1, 0, 1, 2] and spec.head is None
    assert [call.layer for call in describe(SusalornConfig.from_dict(S4)).order] == [0, 1, 2, 1, 2, 3]
    assert [call.layer for call in describe(SusalornConfig.from_dict(S3)).order] == [0, 1, 1, 1]
    shapes = {name: tuple(want.shape) for name, want in expected_tensors(spec).items()}
    assert shapes["l0.mix.dq"] == (40, 64) and shapes["l0.mix.uq"] == (4 * 40, 40)
    assert shapes["l0.mix.dq.norm"] == (40,) and shapes["l0.mix.dkv"] == (64, 64)
    assert shapes["l0.mix.uk"] == (96, 48) and shapes["l0.mix.uv"] == (128, 48)
    assert shapes["l0.mix.sink"] == (4,) and shapes["l0.mix.o"] == (64, 128)
    assert shapes["l1.mix.q"] == (32, 64) and shapes["l1.mix.v.conv"] == (96, 3)
    assert shapes["l1.mix.a1"] == (8, 64) and shapes["l1.mix.a2"] == (64, 8)
    assert shapes["l1.mix.g1"] == (16, 64) and shapes["l1.mix.g2"] == (96, 16)
    assert shapes["l1.mix.dt_bias"] == (64,) and shapes["l1.mix.A_log"] == (4,)
    assert shapes["l0.mlp.e8.up"] == (40, 64) and "l0.mlp.e8.gate" not in shapes
    assert shapes["l0.hc2.mix"] == (4, 4) and shapes["l0.hc1.in"] == (4,)
    assert "l2.hc2.in" not in shapes and "l2.norm2" not in shapes and "head" not in shapes
    needs = cache_entries(spec)
    assert set(needs) == {0, 1, 2, 3, 4}                          # every pass has its own
    assert needs[0] == needs[2] == needs[4] == PagedKeyValues(1, 64, planes=1)
    assert needs[1] == needs[3] == FixedState((4 * 16 * 24 + 3 * (64 + 96),), "float32")


def test_sizes_that_stored_tensors_decide(folders, tmp_path):
    """The inner sizes of the decay and the gate are in no configuration: any stored size loads,
    as long as the pair of matrices agrees on it."""
    from mlx_one_b200.engine.loading import load_model
    from mlx_one_b200.weights import WeightError
    from mlx_one_b200.weights.safetensors_io import write_safetensors

    tensors = plain.read_tensors(folders["S1"] / "model.safetensors")
    bare = json.loads((folders["S1"] / "config.json").read_text())
    assert "decay_rank" not in bare["layers"][1]["mixer"]
    (tmp_path / "config.json").write_text(json.dumps(bare))
    tensors["l1.mix.a1"] = torch.cat([tensors["l1.mix.a1"], tensors["l1.mix.a1"][:3]])
    with pytest.raises(WeightError, match="l1.mix.a2"):
        write_safetensors(tmp_path / "model.safetensors", tensors, {"format": "pt"})
        load_model(tmp_path, "float32", "cpu", PlainOps())
    tensors["l1.mix.a2"] = torch.cat([tensors["l1.mix.a2"], tensors["l1.mix.a2"][:, :3]], dim=1)
    write_safetensors(tmp_path / "model.safetensors", tensors, {"format": "pt"})
    runner, cache = engine(tmp_path, 16, 64)
    (tokens,) = prompts(300, (12,), seed=1)
    got = replay(runner, cache, [([("r", tokens)], ["r"])])["r"]
    assert_rows_close(got, PlainModel(tmp_path).logits(tokens), torch.float32, "a wider decay")
    del tensors["l0.mix.sink"]
    tensors["l0.hc1.mix"] = tensors["l0.hc1.mix"][:3]
    tensors["extra.one"] = torch.zeros(2, dtype=torch.bfloat16)
    write_safetensors(tmp_path / "model.safetensors", tensors, {"format": "pt"})
    with pytest.raises(WeightError) as caught:
        load_model(tmp_path, "float32", "cpu", PlainOps())
    text = str(caught.value)
    assert "l0.mix.sink" in text and "l0.hc1.mix" in text and "extra.one" in text


def test_random_weights_mode(tmp_path):
    from mlx_one_b200.weights import write_random_model

    folder = write_random_model(tmp_path / "drawn", S1, 3)
    runner, cache = engine(folder, 16, 64)
    (tokens,) = prompts(300, (9,), seed=1)
    got = replay(runner, cache, [([("r", tokens)], ["r"])])["r"]
    assert_rows_close(got, PlainModel(folder).logits(tokens), torch.float32, "drawn weights")


# ------------------------------------------------------------------ the plain mechanisms


def test_plain_rotation_by_hand():
    """Fast pairs keep their frequency, slow ones are divided by the factor, both cosine and sine
    carry the amplitude; dimensions behind the rotated ones pass."""
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 10.0, "slow": 1.0}}
    freq, factor = plain.rotation(rot)
    assert freq[0] == 1.0 and freq[3] == pytest.approx(100.0 ** -0.75 / 4)
    assert factor == pytest.approx(0.1 * math.log(4.0) + 1.0)
    x = torch.randn(3, 2, 10, dtype=torch.float64)
    out = plain.rotate_halves(x, torch.tensor([0, 5, 9]), rot)
    assert torch.allclose(out[..., 8:], x[..., 8:])
    assert torch.allclose(out[0, :, :8], x[0, :, :8] * factor)
    u, v = x[1, 0, 1], x[1, 0, 5]
    a = 5 * freq[1]
    assert out[1, 0, 1] == pytest.approx(float(u * math.cos(a) - v * math.sin(a)) * factor)
    assert out[1, 0, 5] == pytest.approx(float(v * math.cos(a) + u * math.sin(a)) * factor)


def test_plain_streams_sink_routing_and_recurrence_by_hand():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=torch.float64)
    mix = torch.tensor([[1.0, 0.5], [0.0, 2.0]], dtype=torch.float64)
    new = plain.write_streams(X, mix, torch.tensor([1.0, -1.0]), torch.tensor([[3.0, 3.0]], dtype=torch.float64))
    assert new[0].tolist() == [[4.0, 5.0]] and new[1].tolist() == [[17.5, 38.0]]    # [from, to]
    weights = plain.softmax_with_sink(torch.zeros(1, 3), torch.tensor([[True, True, False]]),
                                      torch.tensor(math.log(2.0)))
    assert torch.allclose(weights, torch.tensor([[0.25, 0.25, 0.0]]))
    # the second group holds the largest score; its two experts are chosen although the first
    # group's runner-up beats the second of them
    logits = torch.log(torch.tensor([[0.3, 0.25, 0.4, 0.05]], dtype=torch.float64))
    routed = plain.route(logits, {"top": 2, "groups": {"count": 2, "keep": 1}, "scale": 3.0})
    assert torch.allclose(routed, torch.tensor([[0, 0, 0.4, 0.05]], dtype=torch.float64) / 0.45 * 3)
    q = torch.tensor([[[1.0, 0.0]], [[0.0, 1.0]]], dtype=torch.float64)
    k = torch.tensor([[[0.0, 1.0]], [[0.6, 0.8]]], dtype=torch.float64)
    v = torch.tensor([[[2.0]], [[1.0]]], dtype=torch.float64)
    decay = torch.tensor([[[0.5, 0.5]], [[0.9, 0.25]]], dtype=torch.float64)
    out = plain.delta_recurrence(q, k, v, torch.tensor([[1.0], [0.5]], dtype=torch.float64), decay)
    # after the first token S = (0, 2); decayed (0, 0.5); u = 0.5 (1 - 0.4) = 0.3; S = (0.18, 0.74)
    assert out[0].item() == 0.0 and out[1].item() == pytest.approx(0.74)


def test_every_mechanism_moves_the_logits(folders):
    """A sink left out, queries' latents not normed, one decay for all channels, the read-out
    before the write, streams not mixed, a group rule left out, an unscaled rotation: each shows."""
    model = PlainModel(folders["S1"])
    (tokens,) = prompts(300, (40,), seed=2)
    want = model.logits(tokens)

    def moved(change):
        other = PlainModel(folders["S1"])
        change(other)
        return float((other.logits(tokens) - want)[-10:].abs().max())

    def layers(other, kind):
        return [layer for layer in other.config["layers"] if layer["type"] == kind]

    def sinks(other):
        for name in other.weights:
            if name.endswith(".sink"):
                other.weights[name] = other.weights[name] - 50.0

    def scaling(other):
        for layer in layers(other, "latent_attention"):
            del layer["mixer"]["rot"]["scaling"]

    def decays(other):
        other.weights["l1.mix.dt_bias"] = other.weights["l1.mix.dt_bias"].float().mean().expand(64)

    def groups(other):
        other.config["layers"][0]["mlp"]["router"]["groups"]["keep"] = 3

    def scale(other):
        other.config["layers"][0]["mlp"]["router"]["scale"] = 1.0

    def mix(other):
        other.weights["l1.hc1.mix"] = torch.eye(4, dtype=torch.bfloat16)

    def loop(other):
        other.config["loop"]["times"] = 1

    for change in (sinks, scaling, decays, groups, scale, mix, loop):
        assert moved(change) > 0.02, change.__name__


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


@pytest.mark.parametrize("name", ["S1", "S4"])
def test_the_streams_after_every_layer(folders, name):
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], page, 64)
    (tokens,) = prompts(config["vocab"], (19,), seed=2)
    seen = []

    def observe(place, streams, update):
        streams = streams if update is None else update.applied(streams)
        seen.append(streams.sum(1) * (config["streams"] if place < 0 else 1))

    runner.model.observer = observe
    replay(runner, cache, [([("r", tokens)], ["r"])])
    runner.model.observer = None
    states = []
    PlainModel(folders[name]).logits(tokens, states)
    assert len(seen) == len(states) == len(plain.layer_order(config)) + 1
    for place, (got, want) in enumerate(zip(seen, states)):
        assert (got.double() - want).abs().max() < 2e-4, f"after call {place - 1}"


@pytest.mark.parametrize("name", ["S1", "S2", "S5"])
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

    config, _, page = CONFIGS["S1"]
    plain_model = PlainModel(folders["S1"])
    batch = prompts(config["vocab"], (7, 30, 3, 19), seed=8)
    engine_ = Engine(folders["S1"], execution_dtype="float32", ops=PlainOps(), device="cpu",
                     cache_config=CacheConfig(block_size_tokens=page, capacity_tokens=256),
                     batching_config=BatchingConfig(max_sequences=3, prefill_chunk_size=8))
    results = engine_.generate_batch_ids(batch, TextGenerationOptions(max_tokens=6, ignore_eos=True))
    for prompt, result in zip(batch, results):
        assert list(result.token_ids) == plain_model.greedy(prompt, 6)
    engine_.close()

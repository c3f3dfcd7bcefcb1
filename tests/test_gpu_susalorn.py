"""Susalorn on the GPU against the plain implementation: each mechanism alone (parallel streams,
attention over latent rows with a query latent, scaled rotation and sinks, the delta rule with a
decay per key channel, routing in groups, experts without gates), then the engine over whole
requests, decoded tails, portions down to two tokens, mixed batches with pages and slots used
again, keys far away and at page borders, long decoding, replayed graphs and greedy generation."""

import math

import pytest
import torch

import plain_susalorn as plain
from susalorn_models import (CONFIGS, PlainModel, assert_rows_close as assert_close, delta, dense,
                             latent, make_model_dir)
from tiny_models import cut, mixed_schedule, prompts, replay

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
DEVICE = "cuda:0"


@pytest.fixture(scope="module")
def ops():
    from mlx_one_b200.kernels import default_ops
    return default_ops(DEVICE)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("susalorn")
    return {name: make_model_dir(name, root) for name in CONFIGS}


@pytest.fixture(scope="module")
def models(folders):
    return {name: PlainModel(folder) for name, folder in folders.items()}


def engine(folder, dtype, page_size, capacity, max_requests=4):
    from mlx_one_b200.cache import CacheManager
    from mlx_one_b200.engine.loading import load_model
    from mlx_one_b200.engine.runner import Runner

    loaded = load_model(folder, dtype, DEVICE)
    cache = CacheManager(loaded.model.cache_needs, page_size=page_size, capacity_tokens=capacity,
                         max_requests=max_requests, dtype=dtype, device=DEVICE)
    return Runner(loaded.model, cache), cache


def runtime(dtype):
    from mlx_one_b200.kernels import default_ops
    from mlx_one_b200.parts import Runtime
    return Runtime(dtype, torch.device(DEVICE), default_ops(DEVICE))


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEVICE)


def context(portions, histories):
    """A StepContext for requests that bring ``portions`` tokens after ``histories`` tokens."""
    from mlx_one_b200.parts import StepContext

    positions, owner, starts = [], [], [0]
    for r, (n, before) in enumerate(zip(portions, histories)):
        positions += list(range(before, before + n))
        owner += [r] * n
        starts.append(starts[-1] + n)
    return StepContext(tokens=len(positions), requests=len(portions),
                       token_ids=ints([0] * len(positions)), positions=ints(positions),
                       token_request=ints(owner), request_start=ints(starts),
                       history=ints(histories), max_portion=max(portions),
                       max_context=max(p + h for p, h in zip(portions, histories)))


def on(tensor):
    return tensor.to(DEVICE)


def schedule_of(lengths, sizes):
    """Steps of a ragged batch: request r brings its tokens in portions of ``sizes[r]`` (cycled);
    a request that has none left drops out. Yields per step [(request, first, count)]."""
    at = [0] * len(lengths)
    turn = 0
    while any(a < n for a, n in zip(at, lengths)):
        step = []
        for r, n in enumerate(lengths):
            if at[r] < n:
                count = min(sizes[r][turn % len(sizes[r])], n - at[r])
                step.append((r, at[r], count))
                at[r] += count
        turn += 1
        yield step


def page_tables(lengths, page, generator, spare=3):
    """Distinct pages in a random order for requests of the given lengths: (table [requests,
    width] int32 on the host, pages in the pool)."""
    blocks = [-(-n // page) for n in lengths]
    pool = sum(blocks) + spare
    order = torch.randperm(pool, generator=generator).tolist()
    table = torch.full((len(lengths), max(blocks)), -1, dtype=torch.int32)
    for r, count in enumerate(blocks):
        table[r, :count] = torch.tensor([order.pop() for _ in range(count)], dtype=torch.int32)
    return table, pool


# ------------------------------------------------------------------ parallel streams


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("count, tokens, hidden", [
    (1, 3, 64), (2, 5, 36), (3, 300, 192), (4, 7, 1024), (4, 2, 4100), (5, 9, 130), (6, 4, 2048),
    (8, 1, 5000), (11, 3, 72), (16, 2, 260)])
def test_parallel_streams(ops, dtype, count, tokens, hidden):
    """From the one stream at the start through two writes to the sum at the end: every stream, the
    normed reading and the picked rows."""
    from mlx_one_b200.parts import StreamUpdate

    generator = torch.Generator().manual_seed(count)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    x = draw(tokens, hidden)
    weight = 1 + 0.2 * draw(hidden)
    eps = 1e-5
    tight = 2e-5 if dtype == torch.float32 else 2e-2
    X = x.double()[None].repeat(count, 1, 1)
    streams, update = on(x)[:, None], None
    for turn in range(3):
        read, mix, out = draw(count), torch.eye(count) + 0.3 * draw(count, count), draw(count)
        one = turn == 0                     # the streams are still one stream that stands for all
        got, normed = ops.read_streams(streams, update, on(read.sum(0, keepdim=True) if one else read),
                                       on(weight), eps, dtype)
        u = plain.read_streams(X, read.double())
        want = plain.rms_norm(u, weight.double(), eps)
        assert normed.dtype == dtype and (normed.cpu().double() - want).abs().max() < tight * want.abs().max()
        stored = got.cpu().double().transpose(0, 1)
        assert (stored - X[:1] if one else stored - X).abs().max() < 1e-5 * X.abs().max()
        if turn == 2:
            assert got.data_ptr() == streams.data_ptr()          # written in place
        y = draw(tokens, hidden).to(dtype)
        streams, update = got, StreamUpdate(on(y), on(mix.sum(0, keepdim=True) if one else mix), on(out))
        X = plain.write_streams(X, mix.double(), out.double(), y.double())
        if one:
            first = ops.sum_streams(streams, update, None)       # a model of one sublayer
            assert (first.cpu().double() - X.sum(0)).abs().max() < 1e-5 * X.sum(0).abs().max()
    rows = [tokens - 1, 0, tokens // 2]
    picked = ops.sum_streams(streams, update, ints(rows)).cpu().double()
    assert (picked - X.sum(0)[rows]).abs().max() < 2e-5 * X.sum(0).abs().max()
    bare = ops.sum_streams(streams, None, ints([0])).cpu().double()
    assert (bare - streams.cpu().double().sum(1)[:1]).abs().max() < 1e-4


# ------------------------------------------------------------------ attention over latent rows


LATENT_SIZES = [
    # heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden, page, scaling
    (4, 24, 16, 16, 32, 48, 40, 64, 16, (8.0, 64, 16.0, 0.5)),
    (3, 4, 6, 6, 20, 40, 22, 96, 8, None),            # a row of 46 values
    (1, 8, 2, 2, 12, 16, 8, 32, 4, (2.0, 16, 4.0, 1.0)),
    (5, 32, 32, 16, 16, 96, 72, 128, 16, (4.0, 256, 32.0, 1.0)),
    (2, 10, 4, 4, 24, 18, 130, 72, 2, (3.0, 32, 8.0, 2.0)),
    (16, 64, 32, 32, 64, 128, 200, 256, 32, (16.0, 128, 32.0, 1.0)),
    (20, 16, 64, 64, 40, 192, 96, 80, 16, None),      # a row of 256 values, more heads than a tile
]


def latent_case(heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden, scaling, dtype, generator):
    """(the mixer's part, its plain weights and sizes)"""
    from mlx_one_b200.parts import MIXERS, PartSpec

    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "q_rank": q_rank, "scale": 1.7 / math.sqrt(dim + rot_dim), "rot": {"base": 300.0, "dims": dims}}
    keys = ("factor", "original", "fast", "slow")
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(keys, scaling))
    shapes = {"dq": (q_rank, hidden), "uq": (heads * (dim + rot_dim), q_rank),
              "dkv": (kv_rank + rot_dim, hidden), "uk": (heads * dim, kv_rank),
              "uv": (heads * vdim, kv_rank), "o": (hidden, heads * vdim)}
    w = {name: (1.5 * torch.randn(shape, generator=generator) / shape[1] ** 0.5).to(dtype)
         for name, shape in shapes.items()}
    for name, size in (("dq.norm", q_rank), ("dkv.norm", kv_rank)):
        w[name] = (1 + 0.2 * torch.randn(size, generator=generator)).to(dtype)
    w["sink"] = (1 + torch.randn(heads, generator=generator)).to(dtype)
    position = PartSpec("yarn", {"theta": 300.0, "rotary_dim": dims,
                                 **dict(zip(keys, scaling or (None,) * 4))})
    spec = PartSpec("latent_attention", {
        "hidden": hidden, "heads": heads, "head_dim": dim, "rot_dim": rot_dim, "value_dim": vdim,
        "latent": kv_rank, "query_latent": q_rank, "eps": 1e-5, "scale": m["scale"], "gate": False,
        "sink": True, "position": position})
    roles = {"query_down": "dq", "query_norm": "dq.norm", "query_up": "uq", "down": "dkv",
             "down_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "sink": "sink", "out": "o"}
    cls = MIXERS.get("latent_attention")
    part = cls(spec, {role: on(w[name]) for role, name in roles.items()}, runtime(dtype))
    return part, cls.cache_need(spec), {name: t.double() for name, t in w.items()}, m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden, page, scaling",
                         LATENT_SIZES)
def test_latent_attention_part(dtype, heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden, page,
                               scaling):
    """Whole sequences, then the same in portions and single tokens beside each other, against
    the plain mixer that builds every head's keys and values from the latents."""
    from mlx_one_b200.parts import PagedView

    generator = torch.Generator().manual_seed(heads * 100 + dim)
    part, need, wide, m = latent_case(heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden,
                                      scaling, dtype, generator)
    assert need.planes == 1 and need.kv_heads == 1 and need.head_dim == kv_rank + rot_dim
    lengths = (75, 33, 6)
    inputs = [torch.randn(n, hidden, generator=generator).to(dtype).float() for n in lengths]
    want = [plain.latent_attention(x.double(), wide, m, 1e-5, "") for x in inputs]
    table, pool = page_tables(lengths, page, generator)
    tolerance = 2e-4 if dtype == torch.float32 else 0.09
    for sizes in (((1000,),) * 3, ((7, 1, 1, 20, 2), (1,), (2, 3)), ((1,),) * 3):
        kv = torch.full((1, pool, 1, page, kv_rank + rot_dim), 50.0, dtype=dtype, device=DEVICE)
        outputs = [[] for _ in inputs]
        for step in schedule_of(lengths, sizes):
            ctx = context([count for _, _, count in step], [first for _, first, _ in step])
            view = PagedView(kv, on(table[[r for r, _, _ in step]].contiguous()), page, need)
            x = torch.cat([inputs[r][first:first + count] for r, first, count in step]).to(dtype)
            got = part.forward(on(x), ctx, view, True).float().cpu()
            at = 0
            for r, _, count in step:
                outputs[r].append(got[at:at + count])
                at += count
        part.ops.check_errors()
        for r, b in enumerate(want):
            a = torch.cat(outputs[r]).double()
            assert (a - b).abs().max() < tolerance * max(float(b.pow(2).mean().sqrt()), 1.0), \
                f"request {r}, portions {sizes[r]}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("latent_size, rot_dim, dims, page, rank, heads, scaling", [
    (48, 16, 16, 16, 40, 3, (8.0, 64, 16.0, 0.5)), (96, 32, 8, 8, 7, 2, (4.0, 2048, 32.0, 1.0)),
    (512, 64, 64, 16, 1500, 20, None), (18, 4, 4, 2, 12, 1, (40.0, 128, 8.0, 0.25))])
def test_rotation_norms_and_page_write(ops, dtype, latent_size, rot_dim, dims, page, rank, heads, scaling):
    """Positions at the start, at page borders and far away, pages out of order: the stored row,
    the queries' latent and the queries' rotated parts; nothing else in the pages changes."""
    from mlx_one_b200.parts import POSITIONS, PagedKeyValues, PagedView, PartSpec

    generator = torch.Generator().manual_seed(rank)
    rot = {"base": 777.0, "dims": dims}
    keys = ("factor", "original", "fast", "slow")
    if scaling is not None:
        rot["scaling"] = dict(zip(keys, scaling))
    position = POSITIONS.get("yarn")(PartSpec("yarn", {
        "theta": 777.0, "rotary_dim": dims, **dict(zip(keys, scaling or (None,) * 4))}), {}, runtime(dtype))
    portions, histories = [5, 1, 2 * page + 1], [0, 3 * page - 1, 1530]
    ctx = context(portions, histories)
    row = latent_size + rot_dim
    table, pool = page_tables([h + n for n, h in zip(portions, histories)], page, generator)
    kv = torch.full((1, pool, 1, page, row), 9.0, dtype=dtype, device=DEVICE)
    view = PagedView(kv, on(table), page, PagedKeyValues(1, row, planes=1))
    projected = torch.randn(ctx.tokens, rank + row + 3, generator=generator).to(dtype)
    q = torch.randn(ctx.tokens, heads * (5 + rot_dim), generator=generator).to(dtype)
    norm_q, norm_c = (1 + 0.2 * torch.randn(n, generator=generator) for n in (rank, latent_size))
    turn = dict(rot_dim=rot_dim, latent=latent_size, rotary=position.rotary_table(), neighbours=False,
                ctx=ctx, amplitude=position.amplitude())
    small = ops.latent_rows(on(projected), rank=rank, query_norm=on(norm_q), norm_weight=on(norm_c),
                            eps=1e-5, view=view, write=True, **turn)
    queries = torch.full((ctx.tokens, heads, row), 3.0, dtype=dtype, device=DEVICE)
    ops.latent_queries(on(q), queries, heads=heads, head_dim=5, **turn)
    ops.check_errors()
    positions = ctx.positions.cpu()
    wide = projected.double()
    # (32-bit angles: position * frequency is rounded to 1560 * 2^-24 at the far positions)
    bound = 6e-4 if dtype == torch.float32 else 0.03
    want = plain.rms_norm(wide[:, :rank], norm_q.double(), 1e-5)
    assert (small.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 0.03)
    c = plain.rms_norm(wide[:, rank:rank + latent_size], norm_c.double(), 1e-5)
    shared = plain.rotate_halves(wide[:, None, rank + latent_size:rank + row], positions, rot)[:, 0]
    parts = plain.rotate_halves(q.double().view(ctx.tokens, heads, -1)[:, :, 5:], positions, rot)
    assert (queries[:, :, latent_size:].cpu().double() - parts).abs().max() < bound
    assert (queries[:, :, :latent_size] == 3.0).all()
    written = torch.zeros(pool, page, dtype=torch.bool)
    for t, (p, r) in enumerate(zip(positions.tolist(), ctx.token_request.tolist())):
        at = (int(table[r, p // page]), p % page)
        written[at] = True
        stored = kv[0, at[0], 0, at[1]].cpu().double()
        assert (stored - torch.cat([c[t], shared[t]])).abs().max() < bound
    assert (kv[0, :, 0][on(~written)] == 9.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, latent_size, rot_dim", [(8, 64, 16), (3, 40, 6), (16, 128, 32),
                                                        (20, 200, 24), (16, 512, 64), (5, 72, 8)])
def test_sinks_and_a_far_row(ops, dtype, heads, latent_size, rot_dim):
    """One row near the start of 900 matches the last queries by far, and every second head's sink
    outweighs even that one: their outputs are that row's latent, or next to nothing; in a
    prompt's portion, in portions beside single tokens and for single tokens whose keys are cut
    into runs (the sink counts once, whatever the runs). Queries at page borders and tile
    borders, and the first positions, where the sink is most of what there is."""
    from mlx_one_b200.parts import PagedKeyValues, PagedView

    generator = torch.Generator().manual_seed(heads)
    T, page, row = 900, 16, latent_size + rot_dim
    rows = 0.3 * torch.randn(T, row, generator=generator)
    q = 0.3 * torch.randn(T, heads, row, generator=generator)
    rows[3, 5] = 6.0
    rows[3, 6:latent_size] = 1.5
    q[-40:, :, 5] = 8.0
    scale = 0.2
    sinks = 5.0 * torch.rand(heads, generator=generator)
    sinks[1::2] = 12.0
    rows, q = rows.to(dtype), q.to(dtype)
    visible = torch.arange(T)[:, None] >= torch.arange(T)[None, :]
    want = torch.zeros(T, heads, latent_size, dtype=torch.float64)
    for n in range(heads):
        scores = (q[:, n].double() @ rows.double().T) * scale
        want[:, n] = plain.softmax_with_sink(scores, visible, sinks[n].double()) @ rows.double()[:, :latent_size]
    assert want[-1, 0, 6] > 0.4 and want[-1, 1, 6] < 0.4
    table, pool = page_tables((T,), page, generator)
    kv = torch.full((1, pool, 1, page, row), 100.0).to(dtype)
    for t in range(T):
        kv[0, table[0, t // page], 0, t % page] = rows[t]
    need = PagedKeyValues(1, row, planes=1)
    tolerance = 1e-4 if dtype == torch.float32 else 0.04
    for portions, histories in (([40], [T - 40]), ([T], [0]), ([1] * 3, [T - 1, T - 2, T - 3]),
                                ([333, 1, 70], [T - 333, 63, 58]), ([1] * 6, [0, 1, 15, 16, 63, 64]),
                                ([1] * 30, [T - 1 - i for i in range(30)]), ([2, 1], [T - 2, 4]), ([1], [T - 1])):
        ctx = context(portions, histories)
        positions = ctx.positions.tolist()
        view = PagedView(on(kv), on(table.repeat(len(portions), 1).contiguous()), page, need)
        got = ops.latent_attention(on(q[positions]).contiguous(), heads=heads, latent=latent_size,
                                   scale=scale, ctx=ctx, view=view, sinks=on(sinks)).cpu().double()
        assert (got[:, :, :latent_size] - want[positions]).abs().max() < tolerance, str(portions)
    ops.check_errors()


@pytest.mark.parametrize("tokens, heads, head_dim, rot_dim, dims, latent_size", [
    (1, 3, 16, 4, 4, 40), (4, 5, 48, 24, 16, 72), (7, 16, 64, 32, 32, 256), (8, 2, 128, 64, 64, 512),
    (16, 20, 32, 8, 8, 200), (13, 1, 96, 2, 2, 8), (17, 2, 64, 16, 16, 64), (3, 2, 24, 8, 8, 32)])
@pytest.mark.parametrize("neighbours", [False, True])
def test_queries_of_few_tokens_in_one_kernel(ops, tokens, heads, head_dim, rot_dim, dims, latent_size, neighbours):
    """The key up-projection and the rotation of up to 16 tokens in one kernel (more tokens and other
    sizes in two) against the plain products; the queries' rows may be a slice of wider rows."""
    generator = torch.Generator().manual_seed(tokens)
    width = heads * (head_dim + rot_dim)
    q = torch.randn(tokens, width + 24, generator=generator).bfloat16()
    up_k = (torch.randn(heads, latent_size, head_dim, generator=generator) / head_dim ** 0.5).bfloat16()
    inv_freq = torch.rand(dims // 2, generator=generator)
    ctx = context([1] * tokens, [7 * i * i + i for i in range(tokens)])
    queries = torch.full((tokens, heads, latent_size + rot_dim), 9.0, dtype=torch.bfloat16, device=DEVICE)
    ops.latent_absorb(on(q)[:, :width], on(up_k), queries, heads=heads, head_dim=head_dim, rot_dim=rot_dim,
                      latent=latent_size, rotary=(on(inv_freq), dims), neighbours=neighbours, ctx=ctx,
                      amplitude=1.3)
    rows = q[:, :width].double().view(tokens, heads, -1)
    front = torch.einsum("thk,hnk->thn", rows[:, :, :head_dim], up_k.double())
    parts = rows[:, :, head_dim:].clone()
    angle = (ctx.positions.cpu().float()[:, None] * inv_freq[None, :]).double()[:, None, :]
    first = slice(0, dims, 2) if neighbours else slice(0, dims // 2)
    second = slice(1, dims, 2) if neighbours else slice(dims // 2, dims)
    u, v = parts[..., first].clone(), parts[..., second].clone()
    parts[..., first] = 1.3 * (u * torch.cos(angle) - v * torch.sin(angle))
    parts[..., second] = 1.3 * (v * torch.cos(angle) + u * torch.sin(angle))
    got = queries.cpu().double()
    assert (got[:, :, :latent_size] - front).abs().max() < 0.02 * max(1.0, float(front.abs().max()))
    assert (got[:, :, latent_size:] - parts).abs().max() < 0.03


# ------------------------------------------------------------------ the delta rule


DELTA_SIZES = [
    # heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank
    (4, 2, 16, 24, 3, 8, 16), (3, 1, 20, 10, 1, 5, 7), (1, 1, 8, 16, 6, 8, 8), (2, 1, 128, 64, 4, 32, 64),
    (4, 4, 48, 32, 4, 24, 128), (2, 2, 40, 136, 4, 16, 16), (1, 1, 130, 24, 5, 20, 4), (3, 3, 9, 14, 2, 3, 12),
    (2, 2, 256, 40, 4, 12, 260), (6, 2, 128, 128, 4, 128, 128), (2, 1, 33, 66, 4, 16, 8)]


def delta_case(heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank, dtype, seed):
    generator = torch.Generator().manual_seed(seed)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    channels, inner = 2 * kv_heads * dim + heads * vdim, heads * vdim
    up = lambda n: -(-n // 8) * 8
    decay_at = up(channels + heads)
    gate_at = decay_at + up(decay_rank)
    return dict(
        sizes=dict(heads=heads, kv_heads=kv_heads, key_dim=dim, value_dim=vdim, taps=taps),
        decay_columns=(decay_at, decay_at + decay_rank), gate_columns=(gate_at, gate_at + gate_rank),
        width=gate_at + up(gate_rank), channels=channels, inner=inner,
        decay_up=(draw(heads * dim, decay_rank) / decay_rank ** 0.5).to(dtype),
        gate_up=(draw(inner, gate_rank) / gate_rank ** 0.5).to(dtype), conv=0.5 * draw(channels, taps),
        a_log=-1.5 + 0.7 * draw(heads), dt_bias=-1.0 + 1.5 * draw(heads * dim), norm=1 + 0.2 * draw(vdim))


def plain_delta(projected, case, eps):
    """One sequence's mixer from its projected rows on (64-bit)."""
    s, x = case["sizes"], projected.double()
    H, G, D, V = s["heads"], s["kv_heads"], s["key_dim"], s["value_dim"]
    T = x.shape[0]
    mixed = plain.convolve(x[:, :case["channels"]], case["conv"].double())
    qk = G * D
    share = H // G
    q = (plain.unit(mixed[:, :qk].view(T, G, D)) * D ** -0.5).repeat_interleave(share, 1)
    k = plain.unit(mixed[:, qk:2 * qk].view(T, G, D)).repeat_interleave(share, 1)
    beta = torch.sigmoid(x[:, case["channels"]:case["channels"] + H])
    step = plain.softplus(x[:, slice(*case["decay_columns"])] @ case["decay_up"].double().T
                          + case["dt_bias"].double()).view(T, H, D)
    decay = torch.exp(-torch.exp(case["a_log"].double())[None, :, None] * step)
    o = plain.delta_recurrence(q, k, mixed[:, 2 * qk:].view(T, H, V), beta, decay)
    gate = torch.sigmoid(x[:, slice(*case["gate_columns"])] @ case["gate_up"].double().T)
    return plain.rms_norm(o, case["norm"].double(), eps).reshape(T, H * V) * gate


def run_delta(ops, case, inputs, sizes, state, slots, dtype, eps):
    """Requests side by side in portions; returns the outputs per request."""
    from mlx_one_b200.parts import FixedState, StateView

    constants = {name: on(case[name]) for name in ("conv", "a_log", "dt_bias")}
    outputs = [[] for _ in inputs]
    for step in schedule_of([x.shape[0] for x in inputs], sizes):
        ctx = context([count for _, _, count in step], [first for _, first, _ in step])
        view = StateView(state, ints([slots[r] for r, _, _ in step]), FixedState((state.shape[1],), "float32"))
        x = torch.cat([inputs[r][first:first + count] for r, first, count in step])
        got = ops.channel_delta_rule(
            on(x), on(case["decay_up"]), on(case["gate_up"]), decay_columns=case["decay_columns"],
            gate_columns=case["gate_columns"], norm_weight=on(case["norm"]), eps=eps, unit_eps=1e-6,
            ctx=ctx, view=view, write=True, **constants, **case["sizes"]).float().cpu()
        at = 0
        for r, _, count in step:
            outputs[r].append(got[at:at + count])
            at += count
    return [torch.cat(parts).double() for parts in outputs]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", DELTA_SIZES)
def test_channel_delta_rule_alone(ops, dtype, sizes):
    """Requests of unequal length side by side: whole, in portions around the groups of eight
    tokens and the staged sixteen (also shorter than the convolution), and token by token, on
    slots that are zeroed and used again; against one pass of the plain recurrence."""
    from mlx_one_b200.parts import MIXERS, PartSpec

    case = delta_case(*sizes, dtype, sum(sizes))
    eps = 1e-5
    generator = torch.Generator().manual_seed(7)
    lengths = (53, 17, 1, 8, 30)
    inputs = [torch.randn(n, case["width"], generator=generator).to(dtype) for n in lengths]
    want = [plain_delta(x, case, eps) for x in inputs]
    s = case["sizes"]
    size = MIXERS.get("channel_delta").state_size(dict(s))
    state = torch.full((7, size), 5.0, device=DEVICE)
    tolerance = 3e-4 if dtype == torch.float32 else 0.03
    for turn, portions in enumerate((((100,),) * 5, ((7, 1, 9, 16, 2), (1,), (1,), (2, 6), (8, 15, 3)),
                                     ((1,),) * 5, ((2,), (17,), (1,), (3, 1), (31,)))):
        slots = [(r * 3 + turn) % 7 for r in range(5)]
        state[slots] = 0.0
        got = run_delta(ops, case, inputs, portions, state, slots, dtype, eps)
        for r, b in enumerate(want):
            assert (got[r] - b).abs().max() < tolerance, f"request {r} portions {portions[r]}"
    unused = [slot for slot in range(7) if slot not in [(r * 3 + t) % 7 for t in range(4) for r in range(5)]]
    assert all((state[slot] == 5.0).all() for slot in unused)


@pytest.mark.parametrize("dtype", DTYPES)
def test_channels_that_keep_and_channels_that_forget(ops, dtype):
    """Half of the key channels decay by a thousandth a token, half are gone after one: what the
    third token wrote still moves the output 700 tokens later (by decoding and in a prompt), and
    decays that underflow to zero leave no trace of what was there."""
    from mlx_one_b200.parts import MIXERS

    case = delta_case(2, 1, 32, 16, 4, 8, 8, dtype, 5)
    case["decay_up"].zero_()
    case["a_log"].zero_()
    bias = torch.full((2, 32), -7.0)
    bias[:, ::2] = 120.0
    case["dt_bias"] = bias.reshape(-1)
    generator = torch.Generator().manual_seed(9)
    x = torch.randn(700, case["width"], generator=generator).to(dtype)
    x[:, case["channels"]:case["channels"] + 2] = -4.0        # later writes are weak
    x[2, case["channels"]:case["channels"] + 2] = 6.0
    want = plain_delta(x, case, 1e-5)
    changed = x.clone()
    changed[2, 2 * 32:case["channels"]] *= -1.0
    moved = (plain_delta(changed, case, 1e-5)[-1] - want[-1]).abs().max()
    assert moved > 0.05
    size = MIXERS.get("channel_delta").state_size(dict(case["sizes"]))
    for portions in (((1000,),), ((333, 2, 200, 1),), ((1,),)):
        state = torch.zeros(1, size, device=DEVICE)
        (got,) = run_delta(ops, case, [x], portions, state, [0], dtype, 1e-5)
        assert torch.isfinite(got).all()
        assert (got - want).abs().max() < (5e-4 if dtype == torch.float32 else 0.04), str(portions)


# ------------------------------------------------------------------ routed experts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, groups, keep, scale, hidden", [
    (9, 2, 3, 1, 1.5, 64), (6, 4, 3, 3, 2.5, 72), (16, 3, 2, 1, 1.0, 36), (5, 1, None, None, 1.0, 40),
    (3, 3, None, None, 0.7, 130), (64, 8, 8, 3, 2.0, 256), (512, 40, 16, 4, 1.0, 96), (40, 2, 40, 5, 1.0, 33)])
def test_routing_in_groups(ops, dtype, experts, top, groups, keep, scale, hidden):
    generator = torch.Generator().manual_seed(experts)
    x = torch.randn(61, hidden, generator=generator).to(dtype)
    router = 3.0 * torch.randn(experts, hidden, generator=generator) / hidden ** 0.5
    margins = []
    config = {"top": top, "scale": scale}
    if groups:
        config["groups"] = {"count": groups, "keep": keep}
    want = plain.route(x.double() @ router.double().T, config, margins)
    extra = dict(groups=groups, keep=keep, group_score=1) if groups else {}
    got, others = ops.route_general(on(x), on(router), None, experts=experts, identity=0, top=top,
                                    scores="softmax", normalize=True, shared_gate=False, scale=scale, **extra)
    settled = margins[0] > 1e-5
    assert settled.float().mean() > 0.9
    assert ((got.cpu() > 0).sum(1) == top).all()
    assert (got.cpu().double() - want)[settled].abs().max() < 1e-5 * scale
    assert (others[0] == 0).all() and (others[1] == 1).all()
    # equal scores: the lower group, then the lower expert
    even, _ = ops.route_general(on(x[:1]), on(torch.zeros_like(router)), None, experts=experts, identity=0,
                                top=top, scores="softmax", normalize=True, shared_gate=False, **extra)
    assert torch.nonzero(even[0].cpu()).flatten().tolist() == list(range(top))


@pytest.mark.parametrize("score, group_score", [("sigmoid", 2), ("softmax", 3), ("sigmoid", 1)])
def test_group_scores_of_several_experts(ops, score, group_score):
    """The second routing kernel's groups with sums of several scores, against a plain choice."""
    generator = torch.Generator().manual_seed(group_score)
    x = torch.randn(40, 64, generator=generator)
    router = torch.randn(24, 64, generator=generator) / 4
    got, _ = ops.route_general(on(x), on(router), None, experts=24, identity=0, top=4, scores=score,
                               normalize=True, shared_gate=False, groups=6, keep=2, group_score=group_score)
    logits = x.double() @ router.double().T
    s = torch.sigmoid(logits) if score == "sigmoid" else torch.softmax(logits, -1)
    for t in range(40):
        best = s[t].view(6, 4).topk(group_score, -1).values.sum(-1).topk(2).indices.tolist()
        allowed = [e for e in range(24) if e // 4 in best]
        chosen = sorted(allowed, key=lambda e: -float(s[t, e]))[:4]
        expect = torch.zeros(24, dtype=torch.float64)
        expect[chosen] = s[t, chosen] / s[t, chosen].sum()
        assert (got[t].cpu().double() - expect).abs().max() < 1e-5, f"token {t}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden, width, experts, top, groups, keep", [
    (64, 40, 9, 2, 3, 1), (96, 24, 8, 2, 4, 2), (256, 136, 16, 4, 4, 2), (72, 20, 6, 4, 3, 3),
    (128, 304, 4, 1, 1, 1)])
def test_experts_without_gates(dtype, hidden, width, experts, top, groups, keep):
    """One token, a few, enough to be sorted by expert (grouped products): down(relu(up x)^2) of the
    chosen experts, also where an expert gets no token or more than a tile of them."""
    from mlx_one_b200.parts import FEED_FORWARDS, PartSpec

    generator = torch.Generator().manual_seed(width)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    w = {"router": (3.0 * draw(experts, hidden) / hidden ** 0.5).to(dtype)}
    for e in range(experts):
        w[f"e{e}.up"] = (1.5 * draw(width, hidden) / hidden ** 0.5).to(dtype)
        w[f"e{e}.down"] = (draw(hidden, width) / width ** 0.5).to(dtype)
    m = {"router": {"experts": experts, "top": top, "scale": 1.7, "groups": {"count": groups, "keep": keep}}}
    part = FEED_FORWARDS.get("routed")(PartSpec("routed", {
        "hidden": hidden, "width": width, "experts": experts, "top": top, "groups": groups, "keep": keep,
        "group_score": 1, "scale": 1.7, "scores": "softmax", "gated": False, "activation": "relu2"}),
        {name: on(t) for name, t in w.items()}, runtime(dtype))
    wide = {name: t.double() for name, t in w.items()}
    for tokens, shift in ((1, 0.0), (2, 0.0), (7, 0.0), (40, 0.0), (200, 0.0), (450, 2.0)):
        x = draw(tokens, hidden)
        x = (x + shift * wide["router"][1].float() / wide["router"][1].float().norm()).to(dtype)
        margins = []
        want = plain.experts(x.double(), wide, m, "", margins)
        got = part.forward(on(x), None).cpu().double()
        part.ops.check_errors()
        settled = margins[0] > (1e-5 if dtype == torch.float32 else 1e-4)
        tolerance = 2e-4 if dtype == torch.float32 else 0.03
        error = (got - want)[settled].abs().max() / max(1.0, float(want.abs().max()))
        assert error < tolerance, f"{tokens} tokens: {error}"


# ------------------------------------------------------------------ the engine


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_requests_and_first_tokens(folders, models, name, dtype):
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], dtype, page, 256)
    for tokens in prompts(config["vocab"], (150, 1, 2, 5), seed=3):
        got = replay(runner, cache, [([("w", tokens)], ["w"])])["w"]
        assert_close(got, models[name].logits(tokens), dtype, f"{name} whole {len(tokens)}")


def test_the_streams_after_every_layer(folders, models):
    for name in ("S1", "S4"):
        config, _, page = CONFIGS[name]
        runner, cache = engine(folders[name], torch.float32, page, 64)
        (tokens,) = prompts(config["vocab"], (19,), seed=2)
        seen = []

        def observe(place, streams, update):
            streams = streams if update is None else update.applied(streams)
            seen.append(streams.sum(1) * (config["streams"] if place < 0 else 1))

        runner.model.observer = observe
        replay(runner, cache, [([("r", tokens)], ["r"])])
        runner.model.observer = None
        states = []
        models[name].logits(tokens, states)
        assert len(seen) == len(states) == len(plain.layer_order(config)) + 1
        for place, (got, want) in enumerate(zip(seen, states)):
            # (a step's rows may be padded to a shape that is replayed)
            got = got[:len(tokens)].cpu().double()
            assert (got - want).abs().max() < 5e-4, f"{name} after call {place - 1}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prefill_against_token_by_token(folders, models, name, dtype):
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], dtype, page, 128)
    (tokens,) = prompts(config["vocab"], (70,), seed=4)
    want = models[name].logits(tokens)
    whole = replay(runner, cache, [([("w", tokens)], ["w"])])["w"]
    steps = [([("d", [token])], []) for token in tokens]
    steps[-1] = (steps[-1][0], ["d"])
    single = replay(runner, cache, steps)["d"]
    assert_close(whole, want, dtype, f"{name} whole")
    assert_close(single, want, dtype, f"{name} token by token")
    if dtype == torch.float32 and (want.margin > 1e-4).all():
        assert (whole - single).abs().max() < 5e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_changing_size(folders, models, name, dtype):
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], dtype, page, 192)
    (tokens,) = prompts(config["vocab"], (170,), seed=5)
    want = models[name].logits(tokens)
    for sizes in ((7, 2, 40, 3, 1, 1), (2,), (64, 1), (33, 31)):
        steps = [([("p", part)], []) for part in cut(tokens, sizes)]
        steps[-1] = (steps[-1][0], ["p"])
        assert_close(replay(runner, cache, steps)["p"], want, dtype, f"{name} portions {sizes}")
    assert not cache.requests()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(folders, models, name, dtype):
    config, _, page = CONFIGS[name]
    lengths = (150, 64, 23, 50, 17, 9, 2, 1, 40)
    requests = dict(enumerate(prompts(config["vocab"], lengths, seed=6)))
    runner, cache = engine(folders[name], dtype, page, 4 * 192, max_requests=4)
    got = replay(runner, cache, mixed_schedule(requests))
    for key, tokens in requests.items():
        want = models[name].logits(tokens)
        assert_close(got[key], want, dtype, f"{name} mixed request {key}")
        alone = replay(runner, cache, [([("alone", tokens)], ["alone"])])["alone"]
        if dtype == torch.float32 and (want.margin > 1e-4).all():
            assert (alone - got[key]).abs().max() < 5e-4, f"{name} request {key} beside others"
    assert not cache.requests()
    cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["S1", "S4"])
def test_steps_of_a_repeated_shape_are_replayed(folders, models, name, dtype):
    """Single tokens of three requests step after step: the runner captures the step's shape and
    replays it with other tokens, positions, tables and slots; the logits stay the plain model's."""
    config, _, page = CONFIGS[name]
    runner, cache = engine(folders[name], dtype, page, 512, max_requests=3)
    requests = dict(zip("abc", prompts(config["vocab"], (60, 41, 52), seed=7)))
    steps = [([(key, tokens[:20]) for key, tokens in requests.items()], [])]
    for i in range(20, 60):
        live = [(key, [tokens[i]]) for key, tokens in requests.items() if i < len(tokens)]
        steps.append((live, [key for key, tokens in requests.items() if i == len(tokens) - 1]))
    got = replay(runner, cache, steps)
    assert runner.graph_replays > 20
    for key, tokens in requests.items():
        assert_close(got[key], models[name].logits(tokens), dtype, f"{name} request {key}")
    assert not cache.requests()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_far_rows(tmp_path, dtype):
    """A prompt in portions that cut pages and groups of tokens, then 260 tokens decoded one by
    one; the third token still moves the last logits (the plain model says by how much)."""
    config = {"architecture": "Susalorn", "vocab": 200, "width": 64, "norm": {"eps": 1e-5}, "streams": 2,
              "layers": [latent(4, 16, 8, 16, 32, 24, 0.3, dense(128), scaling=(4.0, 128, 16.0, 1.0)),
                         delta(4, 2, 16, 16, 4, dense(128)),
                         latent(2, 24, 16, 40, 56, 40, 0.25, None, base=50000.0),
                         delta(2, 1, 32, 24, 3, dense(96))],
              "loop": {"start": 1, "stop": 3, "times": 2}}
    folder = make_model_dir("S1", tmp_path, config)
    model = PlainModel(folder)
    (tokens,) = prompts(config["vocab"], (640,), seed=21)
    want = model.logits(tokens)
    changed = list(tokens)
    changed[2] = (changed[2] + 1) % config["vocab"]
    moved = (model.logits(changed)[-1] - want[-1]).abs().max()
    runner, cache = engine(folder, dtype, 16, 640, max_requests=2)
    sizes = [209, 129, 2, 3, 37] + [1] * 260
    assert sum(sizes) == len(tokens)
    steps, at = [], 0
    for size in sizes:
        steps.append(([("long", tokens[at:at + size])], []))
        at += size
    steps[-1] = (steps[-1][0], ["long"])
    got = replay(runner, cache, steps)["long"]
    assert_close(got, want, dtype, "long decoding")
    if dtype == torch.float32:
        assert moved > 1e-3 and moved > 20 * (got[-1].cpu() - want[-1]).abs().max(), \
            "the first tokens no longer show at the end"


def test_greedy_generation_through_the_entry_point(folders, models):
    from mlx_one_b200 import BatchingConfig, CacheConfig, Engine, TextGenerationOptions

    for name, dtype in (("S1", "float32"), ("S4", "float32"), ("S2", "bfloat16")):
        config, _, page = CONFIGS[name]
        engine_ = Engine(folders[name], execution_dtype=dtype,
                         cache_config=CacheConfig(block_size_tokens=page, capacity_tokens=512),
                         batching_config=BatchingConfig(max_sequences=3, prefill_chunk_size=16))
        batch = prompts(config["vocab"], (7, 30, 3, 19, 12), seed=8)
        results = engine_.generate_batch_ids(batch, TextGenerationOptions(max_tokens=12, ignore_eos=True))
        if dtype == "float32":
            for prompt, result in zip(batch, results):
                assert list(result.token_ids) == models[name].greedy(prompt, 12)
        else:
            assert all(len(result.token_ids) == 12 for result in results)
        engine_.close()


def test_command_line_and_trace_replay(folders, models, tmp_path):
    """`mlx-one generate` with token ids (greedy against the plain model) and `trace_run` as a
    process: steps on standard input, logits files out, requests ended and their slots used
    again."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    root = Path(__file__).resolve().parent.parent
    folder = folders["S4"]
    greedy = subprocess.run([sys.executable, str(root / "bin" / "mlx-one"), "generate", str(folder),
                             "5 17 3 200", "--token-ids", "--max-tokens", "6", "--dtype", "float32"],
                            capture_output=True, text=True, timeout=600)
    assert greedy.returncode == 0, greedy.stderr
    assert [int(t) for t in greedy.stdout.split()] == models["S4"].greedy([5, 17, 3, 200], 6)

    vocab = CONFIGS["S4"][0]["vocab"]
    a, b, c = prompts(vocab, (21, 9, 30), seed=17)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:8], "want": [0, 7]},
                                     {"id": "b", "tokens": b, "want": [8]}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": a[8:20], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[20:], "want": [0]},
                                     {"id": "c", "tokens": c[:2], "want": [1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c[2:], "want": [27]}], "end": ["c"]}]
    out = tmp_path / "logits"
    done = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder),
                           "--dtype", "float32", "--out", str(out), "--max-tokens", "128",
                           "--max-requests", "2"],
                          input="".join(json.dumps(step) + "\n" for step in steps),
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr
    assert [line for line in done.stdout.split("\n") if line.startswith("done")] == \
        [f"done {i}" for i in range(4)]
    read = lambda step, rows: torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4")).view(rows, vocab)
    assert not (out / "1.f32").exists()
    wa, wb, wc = (models["S4"].logits(t) for t in (a, b, c))
    close = lambda got, want: (got - want).abs().max() < 5e-4
    assert close(read(0, 3), torch.stack([wa[0], wa[7], wb[8]]))
    assert close(read(2, 2), torch.stack([wa[20], wc[1]]))
    assert close(read(3, 1), wc[29:30])

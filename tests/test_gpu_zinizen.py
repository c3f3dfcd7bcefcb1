"""Zinizen on the GPU against the plain implementation: each mechanism alone (layer norms around the
adds, norms over whole rows with a temperature and mixed values, capped and distance-biased scores,
latent attention with a gate per head, the gated linear recurrence, clamped experts), then the
engine over whole requests, decoded tails, portions down to two tokens, mixed batches with pages
and slots used again, keys far away and at page borders, long decoding, replayed graphs and greedy
generation."""

import math

import pytest
import torch

import plain_zinizen as plain
from test_gpu_susalorn import context, engine, ints, on, page_tables, runtime, schedule_of
from tiny_models import cut, mixed_schedule, prompts, replay
from zinizen_models import (CONFIGS, PlainModel, assert_rows_close as assert_close, attention, bigram,
                            dense, latent, make_model_dir, rglru)

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
DEVICE = "cuda:0"


@pytest.fixture(scope="module")
def ops():
    from mlx_one_b200.kernels import default_ops
    return default_ops(DEVICE)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zinizen")
    return {name: make_model_dir(name, root) for name in CONFIGS}


@pytest.fixture(scope="module")
def models(folders):
    return {name: PlainModel(folder) for name, folder in folders.items()}


# ------------------------------------------------------------------ norms of the stream


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, hidden", [
    (1, 64), (3, 36), (5, 257), (2, 1000), (7, 4096), (3, 8192), (2, 8200), (2, 10001), (1600, 200),
    (1540, 512), (1536, 1024), (1100, 2048), (1024, 6144), (40, 5120)])
def test_norms_around_an_add(ops, dtype, rows, hidden):
    """Layer norms and root-mean-square norms ahead of the next part, after nothing, after a plain
    output with a factor and after an output that is normed itself. The values have a mean far
    from zero, so that a variance taken about zero would show."""
    from mlx_one_b200.parts import NormedUpdate

    generator = torch.Generator().manual_seed(rows + hidden)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    eps, post_eps = 1e-5, 3e-4
    x = 20.0 + draw(rows, hidden)
    y = (3.0 - 2.0 * draw(rows, hidden)).to(dtype)
    w, b, pw, pb = 1 + 0.3 * draw(hidden), draw(hidden), 1 + 0.3 * draw(hidden), draw(hidden)
    rms = lambda v, weight, e: plain.rms_norm(v, weight.double(), e)
    layer = lambda v, weight, bias, e: plain.layer_norm(v, weight.double(), bias.double(), e)
    wide = y.double()
    cases = [(None, 1.0, x.double()), (on(y), 0.7, x.double() + 0.7 * wide),
             (NormedUpdate(on(y), on(pw), on(pb), post_eps), 1.0,
              x.double() + layer(wide, pw, pb, post_eps)),
             (NormedUpdate(on(y), on(pw), None, post_eps), 1.0, x.double() + rms(wide, pw, post_eps))]
    for delta, factor, stream in cases:
        for bias in (b, None):
            residual = on(x).clone()
            got = ops.add_norm(residual, delta, on(w), None if bias is None else on(bias), eps, dtype,
                               delta_scale=factor)
            want = rms(stream, w, eps) if bias is None else layer(stream, w, bias, eps)
            assert (residual.cpu().double() - stream).abs().max() < 2e-5
            bound = 1e-4 if dtype == torch.float32 else 0.02 * max(1.0, float(want.abs().max()))
            assert got.dtype == dtype and (got.cpu().double() - want).abs().max() < bound


# ------------------------------------------------------------------ queries, keys and values


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, page, temp, mix, rotary", [
    (4, 2, 32, 16, 16, (0.4, 16), 0.3, 0), (3, 1, 20, 28, 8, (1.0, 1), None, 0), (1, 1, 16, 16, 4, None, 0.8, 0),
    (6, 2, 128, 128, 2, (0.25, 64), -0.4, 0), (8, 8, 64, 48, 32, (0.5, 2.5), 1.0, 0),
    (4, 2, 32, 32, 16, (0.4, 16), 0.3, 16), (2, 2, 10, 14, 16, None, None, 0)])
def test_norm_over_rows_temperature_and_mixed_values(ops, dtype, heads, kv_heads, dim, vdim, page, temp,
                                                    mix, rotary):
    """Positions at the start, on both sides of a step of the temperature, at page borders and far
    away, pages out of order: the queries, and the keys and values in the pages; nothing else in
    them changes. One head is far larger than the others, so that a norm per head would show."""
    from mlx_one_b200.parts import PagedKeyValues, PagedView

    generator = torch.Generator().manual_seed(heads * dim)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    portions, histories = [5, 1, 2 * page + 1, 3], [0, 3 * page - 1, 1530, 61]
    ctx = context(portions, histories)
    T, row = ctx.tokens, max(dim, vdim)
    q_size, k_size, v_size = heads * dim, kv_heads * dim, kv_heads * vdim
    projected = draw(T, q_size + k_size + v_size + 5)
    projected[:, :dim] *= 6.0
    projected[:, q_size:q_size + dim] *= 4.0
    projected, first = projected.to(dtype), draw(T, v_size + 3).to(dtype)
    qw, kw = 1 + 0.3 * draw(q_size), 1 + 0.3 * draw(k_size)
    table, pool = page_tables([h + n for n, h in zip(portions, histories)], page, generator)
    kv = torch.full((2, pool, kv_heads, page, row), 9.0, dtype=dtype, device=DEVICE)
    view = PagedView(kv, on(table), page, PagedKeyValues(kv_heads, row))
    inv_freq = torch.rand(max(rotary // 2, 1), generator=generator) / 50
    got = ops.qk_norm_rope_store(
        on(projected)[:, :q_size + k_size + v_size], heads=heads, kv_heads=kv_heads, head_dim=dim,
        q_weight=on(qw), k_weight=on(kw), eps=1e-5, rotary=(on(inv_freq), rotary) if rotary else None,
        ctx=ctx, view=view, write=True, value_dim=vdim, norm_rows=True, temperature=temp,
        value_mix=None if mix is None else (mix, on(first)[:, :v_size]))
    ops.check_errors()
    wide, positions = projected.double(), ctx.positions.cpu()

    def turned(x):
        if not rotary:
            return x
        angle = (positions.float()[:, None] * inv_freq[None, :]).double()[:, None, :]
        u, v = x[..., :rotary // 2], x[..., rotary // 2:rotary]
        return torch.cat([u * torch.cos(angle) - v * torch.sin(angle),
                          v * torch.cos(angle) + u * torch.sin(angle), x[..., rotary:]], -1)

    q = plain.rms_norm(wide[:, :q_size], qw.double(), 1e-5).view(T, heads, dim)
    if temp is not None:
        q = q * plain.temperature(positions.tolist(), dict(zip(("coef", "every"), temp)),
                                  torch.float64)[:, None, None]
    k = plain.rms_norm(wide[:, q_size:q_size + k_size], kw.double(), 1e-5).view(T, kv_heads, dim)
    v = wide[:, q_size + k_size:q_size + k_size + v_size]
    if mix is not None:
        v = plain.mix_values(v, first.double()[:, :v_size], mix)
    q, k, v = turned(q), turned(k), v.view(T, kv_heads, vdim)
    bound = 5e-5 if dtype == torch.float32 else 0.05
    assert (got[..., :dim].cpu().double() - q).abs().max() < bound * max(1.0, float(q.abs().max()) / 4)
    assert (got[..., dim:] == 0).all()
    written = torch.zeros(pool, page, dtype=torch.bool)
    for t, (p, r) in enumerate(zip(positions.tolist(), ctx.token_request.tolist())):
        at = (int(table[r, p // page]), p % page)
        written[at] = True
        for plane, want, size in ((0, k, dim), (1, v, vdim)):
            stored = kv[plane, at[0], :, at[1]].cpu().double()
            assert (stored[:, :size] - want[t]).abs().max() < bound and (stored[:, size:] == 0).all()
    assert (kv.transpose(2, 3)[:, on(~written)] == 9.0).all()


# ------------------------------------------------------------------ shaped scores


def plain_scores(q, k, v, scale, cap, slope):
    return plain.biased_attention(q.double(), k.double(), v.double(), scale, cap, slope.double())


SHAPED = [
    # heads, kv_heads, row size, cap, slopes, scale
    (4, 2, 64, 6.0, True, 0.4), (8, 2, 64, None, True, 0.3), (3, 1, 32, 4.0, True, 0.5),
    (2, 2, 128, 50.0, True, 0.2), (16, 4, 64, 2.0, True, 0.5), (5, 5, 112, 3.0, False, 0.3),
    (6, 1, 20, 5.0, True, 0.5), (10, 5, 48, 20.0, True, 0.25), (1, 1, 16, 8.0, True, 0.6)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, cap, sloped, scale", SHAPED)
def test_capped_and_distance_biased_scores(ops, dtype, heads, kv_heads, dim, cap, sloped, scale):
    """One key near the start of 700 matches the last queries by far and is worth 45 in its values,
    several near ones match by less: what the far one is worth depends on the cap and on the
    distance, head by head. In whole prompts, portions beside single tokens, and single tokens at
    page and tile borders whose keys are cut into runs."""
    from mlx_one_b200.parts import PagedKeyValues, PagedView

    generator = torch.Generator().manual_seed(heads * 7 + dim)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    T, page = 700, 16
    q, k, v = 0.4 * draw(T, heads, dim), 0.4 * draw(T, kv_heads, dim), 0.5 * draw(T, kv_heads, dim)
    q[-50:, :, 1] = 5.0
    k[5, :, 1], v[5] = 9.0, 45.0
    k[T - 90:T - 60:7, :, 1] = 1.5
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    slope = plain.slopes(heads, torch.float32) * 0.25 if sloped else torch.zeros(heads)
    want = plain_scores(q, k, v, scale, cap, slope)
    near = plain_scores(q[8:], k[8:], v[8:], scale, cap, slope)         # without the far key
    if float(slope.min()) * T < 15:
        assert (want[-1] - near[-1]).abs().max() > 0.2                   # it shows
    table, pool = page_tables((T,), page, generator)
    kv = torch.full((2, pool, kv_heads, page, dim), 100.0).to(dtype)
    for t in range(T):
        kv[0, table[0, t // page], :, t % page] = k[t]
        kv[1, table[0, t // page], :, t % page] = v[t]
    need = PagedKeyValues(kv_heads, dim)
    shape = dict(score_cap=cap or 0.0, slopes=on(slope) if sloped else None,
                 least_slope=float(slope.min()) if sloped else 0.0)
    tolerance = 2e-4 if dtype == torch.float32 else 0.04
    for portions, histories in (([50], [T - 50]), ([T], [0]), ([1] * 3, [T - 1, T - 2, T - 3]),
                                ([333, 1, 70], [T - 333, 63, 58]), ([1] * 8, [0, 1, 15, 16, 31, 32, 63, 64]),
                                ([1] * 30, [T - 1 - i for i in range(30)]), ([2, 1], [T - 2, 4]), ([1], [T - 1]),
                                ([1, 1, 40], [T - 1, 5, 100])):
        ctx = context(portions, histories)
        if portions == [1, 1, 40]:
            ctx.leading_single = 2
        positions = ctx.positions.tolist()
        view = PagedView(on(kv), on(table.repeat(len(portions), 1).contiguous()), page, need)
        got = ops.paged_attention(on(q[positions]).contiguous(), heads=heads, kv_heads=kv_heads,
                                  head_dim=dim, scale=scale, window=None, ctx=ctx, view=view, **shape)
        got = got.view(len(positions), heads, dim).cpu().double()
        bound = tolerance * torch.clamp(want[positions].abs() / 3, min=1.0)
        assert ((got - want[positions]).abs() < bound).all(), str(portions)
    ops.check_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim", [(8, 2, 64), (16, 16, 128), (12, 3, 32)])
def test_keys_beyond_the_reach_of_a_steep_slope(ops, dtype, heads, kv_heads, dim):
    """Slopes so steep that the kernels leave far keys out: the result is that of all keys, also on
    both sides of the borders at which a key is left out; what a left-out page holds (values that
    are huge, but finite) does not matter."""
    from mlx_one_b200.parts import PagedKeyValues, PagedView

    generator = torch.Generator().manual_seed(dim)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    T, page, cap, scale = 900, 16, 1.5, 0.4
    q, k, v = draw(T, heads, dim), draw(T, kv_heads, dim), draw(T, kv_heads, dim)
    v[:100] = 1e4
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    slope = 2.0 * plain.slopes(heads, torch.float32)
    want = plain_scores(q, k, v, scale, cap, slope)
    assert float((2 * cap + 88) / slope.max()) < 150
    table, pool = page_tables((T,), page, generator)
    kv = torch.zeros((2, pool, kv_heads, page, dim)).to(dtype)
    for t in range(T):
        kv[0, table[0, t // page], :, t % page] = k[t]
        kv[1, table[0, t // page], :, t % page] = v[t]
    shape = dict(score_cap=cap, slopes=on(slope), least_slope=float(slope.min()))
    edges = sorted({min(T - 1, 100 + int((2 * cap + 88) / float(s)) + d) for s in slope for d in (-30, -1, 0, 1, 30)})
    for portions, histories in (([T], [0]), ([1] * len(edges), edges), ([300], [T - 300]), ([1], [T - 1])):
        ctx = context(portions, histories)
        positions = ctx.positions.tolist()
        view = PagedView(on(kv), on(table.repeat(len(portions), 1).contiguous()), page,
                         PagedKeyValues(kv_heads, dim))
        got = ops.paged_attention(on(q[positions]).contiguous(), heads=heads, kv_heads=kv_heads,
                                  head_dim=dim, scale=scale, window=None, ctx=ctx, view=view, **shape)
        got = got.view(len(positions), heads, dim).cpu().double()
        bound = (3e-4 if dtype == torch.float32 else 0.04) * torch.clamp(want[positions].abs(), min=1.0)
        assert ((got - want[positions]).abs() < bound).all(), str(portions)
    ops.check_errors()


# ------------------------------------------------------------------ whole mixers as parts


def attention_case(m, hidden, mix, dtype, generator):
    from mlx_one_b200.architectures.zinizen import _attention
    from mlx_one_b200.config.zinizen import AttentionMixer
    from mlx_one_b200.parts import MIXERS

    spec = _attention(AttentionMixer.from_dict(m, ""), hidden, 1e-5, mix)
    cls = MIXERS.get("attention")
    w, local = {}, {}
    for name, want in cls.tensors(spec).items():
        values = torch.randn(want.shape, generator=generator)
        if len(want.shape) == 2:
            values = 1.5 * values / want.shape[1] ** 0.5
        elif want.init == "norm":
            values = 1 + 0.2 * values
        elif not want.shape:
            values = torch.tensor(0.6)
        local[name] = values.to(dtype)
        w[spec.names[name]] = local[name].double()
    part = cls(spec, {name: on(t) for name, t in local.items()}, runtime(dtype))
    return part, cls.cache_need(spec), w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, hidden, page, cap, temp", [
    (4, 2, 32, 16, 64, 16, 8.0, (0.4, 16)), (3, 1, 20, 28, 52, 8, None, None), (8, 2, 64, 48, 128, 16, 30.0, (0.3, 32)),
    (1, 1, 16, 16, 36, 4, 2.0, (1.0, 1)), (6, 2, 128, 128, 72, 2, 12.0, (0.25, 50)), (5, 5, 48, 64, 96, 64, 9.0, None)])
def test_attention_parts_that_share_values(dtype, heads, kv_heads, dim, vdim, hidden, page, cap, temp):
    """Two mixers in a row, the second mixing its values with the first's: whole sequences, portions
    and single tokens side by side, against the plain mixers."""
    from mlx_one_b200.parts import PagedView

    generator = torch.Generator().manual_seed(heads + dim)
    m = attention(heads, kv_heads, dim, vdim, 1.5 / math.sqrt(dim), None, cap, temp, True)["mixer"]
    first, need, w1 = attention_case(m, hidden, "first", dtype, generator)
    later, _, w2 = attention_case(m, hidden, "later", dtype, generator)
    lengths = (75, 33, 6)
    inputs = [torch.randn(n, hidden, generator=generator).to(dtype).float() for n in lengths]
    want = []
    for x in inputs:
        shared = {}
        a = plain.attention(x.double(), w1, m, 1e-5, "", shared)
        b = plain.attention(x.flip(1).double(), w2, m, 1e-5, "", shared)
        want.append(torch.cat([a, b], 1))
    table, pool = page_tables(lengths, page, generator)
    tolerance = 3e-4 if dtype == torch.float32 else 0.09
    for sizes in (((1000,),) * 3, ((7, 1, 1, 20, 2), (1,), (2, 3)), ((1,),) * 3):
        caches = [torch.full((2, pool, kv_heads, page, need.head_dim), 50.0, dtype=dtype, device=DEVICE)
                  for _ in range(2)]
        outputs = [[] for _ in inputs]
        for step in schedule_of(lengths, sizes):
            ctx = context([count for _, _, count in step], [at for _, at, _ in step])
            tables = on(table[[r for r, _, _ in step]].contiguous())
            x = torch.cat([inputs[r][at:at + count] for r, at, count in step]).to(dtype)
            a = first.forward(on(x), ctx, PagedView(caches[0], tables, page, need), True)
            b = later.forward(on(x.flip(1).contiguous()), ctx, PagedView(caches[1], tables, page, need), True)
            got = torch.cat([a, b], 1).float().cpu()
            at = 0
            for r, _, count in step:
                outputs[r].append(got[at:at + count])
                at += count
        first.ops.check_errors()
        for r, b in enumerate(want):
            a = torch.cat(outputs[r]).double()
            assert (a - b).abs().max() < tolerance * max(float(b.pow(2).mean().sqrt()), 1.0), \
                f"request {r}, portions {sizes[r]}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rot_dim, dims, vdim, kv_rank, q_rank, hidden, page", [
    (3, 24, 8, 8, 32, 48, 40, 64, 16), (2, 6, 4, 2, 10, 18, 22, 52, 8), (1, 8, 2, 2, 12, 16, 8, 36, 4),
    (5, 32, 32, 32, 48, 128, 64, 128, 16), (17, 16, 16, 16, 24, 96, 32, 80, 32), (8, 64, 32, 32, 64, 512, 128, 256, 16)])
def test_latent_attention_with_a_gate_per_head(dtype, heads, dim, rot_dim, dims, vdim, kv_rank, q_rank,
                                               hidden, page):
    from mlx_one_b200.architectures.zinizen import _latent
    from mlx_one_b200.config.zinizen import LatentMixer
    from mlx_one_b200.parts import MIXERS, PagedView

    generator = torch.Generator().manual_seed(heads * 100 + dim)
    m = latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, 1.7 / math.sqrt(dim + rot_dim), None, 300.0, dims)["mixer"]
    spec = _latent(LatentMixer.from_dict(m, ""), hidden, 1e-5)
    cls = MIXERS.get("latent_attention")
    w, local = {}, {}
    for name, shape in cls.tensors(spec).items():
        values = torch.randn(shape.shape, generator=generator)
        values = 1 + 0.2 * values if shape.init == "norm" else 1.5 * values / shape.shape[1] ** 0.5
        local[name] = values.to(dtype)
        w[spec.names[name]] = local[name].double()
    assert w["g"].shape == (heads, hidden)
    part, need = cls(spec, {name: on(t) for name, t in local.items()}, runtime(dtype)), cls.cache_need(spec)
    lengths = (75, 33, 6)
    inputs = [torch.randn(n, hidden, generator=generator).to(dtype).float() for n in lengths]
    want = [plain.latent_attention(x.double(), w, m, 1e-5, "") for x in inputs]
    table, pool = page_tables(lengths, page, generator)
    tolerance = 3e-4 if dtype == torch.float32 else 0.09
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


# ------------------------------------------------------------------ the gated recurrence


def recurrence_case(width, blocks, dtype, seed, lam=-3.5):
    generator = torch.Generator().manual_seed(seed)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    part = width // blocks
    return dict(ra=(2.0 * draw(blocks, part, part) / part ** 0.5).to(dtype),
                ri=(2.0 * draw(blocks, part, part) / part ** 0.5).to(dtype), ra_b=0.5 * draw(blocks, part),
                ri_b=0.5 * draw(blocks, part), lam=lam + 1.5 * draw(width))


def plain_recurrence(u, y, case):
    wide = {name: t.double() for name, t in case.items()}
    u = u.double()
    r = torch.sigmoid(plain.block_products(u, wide["ra"], wide["ra_b"]))
    i = torch.sigmoid(plain.block_products(u, wide["ri"], wide["ri_b"]))
    return plain.linear_recurrence(u, r, i, wide["lam"]) * plain.gelu_tanh(y.double())


def run_recurrence(ops, case, inputs, gates_in, sizes, state, slots):
    from mlx_one_b200.parts import FixedState, StateView

    gates = on(torch.cat([case["ra"], case["ri"]], 1).contiguous())
    bias = on(torch.cat([case["ra_b"], case["ri_b"]], 1).contiguous())
    rate = on((-8 * torch.nn.functional.softplus(case["lam"].double())).float())
    outputs = [[] for _ in inputs]
    for step in schedule_of([x.shape[0] for x in inputs], sizes):
        ctx = context([count for _, _, count in step], [first for _, first, _ in step])
        view = StateView(state, ints([slots[r] for r, _, _ in step]), FixedState((state.shape[1],), "float32"))
        u = torch.cat([inputs[r][first:first + count] for r, first, count in step])
        y = torch.cat([gates_in[r][first:first + count] for r, first, count in step])
        wider = on(torch.cat([y, y[:, :4]], 1))                       # (y is a slice of wider rows)
        got = ops.gated_recurrence(on(u), wider[:, :u.shape[1]], gates=gates, gate_bias=bias, rate=rate,
                                   ctx=ctx, view=view, write=True).float().cpu()
        at = 0
        for r, _, count in step:
            outputs[r].append(got[at:at + count])
            at += count
    return [torch.cat(parts).double() for parts in outputs]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, blocks", [(96, 3), (35, 7), (8, 1), (192, 3), (24, 24), (64, 8), (520, 2),
                                           (1024, 2), (40, 2), (132, 11)])
def test_gated_recurrence_alone(ops, dtype, width, blocks):
    """Requests of unequal length side by side: whole (cut into chunks), in portions around a chunk's
    length, and token by token (the gates' product in the kernel), on slots that are zeroed and used
    again; against one pass of the plain recurrence."""
    case = recurrence_case(width, blocks, dtype, width)
    generator = torch.Generator().manual_seed(7)
    lengths = (150, 33, 1, 16, 70)
    inputs = [torch.randn(n, width, generator=generator).to(dtype) for n in lengths]
    gates_in = [torch.randn(n, width, generator=generator).to(dtype) for n in lengths]
    want = [plain_recurrence(x, y, case) for x, y in zip(inputs, gates_in)]
    state = torch.full((7, width), 5.0, device=DEVICE)
    tolerance = 2e-4 if dtype == torch.float32 else 0.03
    for turn, portions in enumerate((((1000,),) * 5, ((40, 1, 63, 16, 2), (1,), (1,), (2, 6), (33, 15, 3)),
                                     ((1,),) * 5, ((2,), (17,), (1,), (3, 1), (32,)))):
        slots = [(r * 3 + turn) % 7 for r in range(5)]
        state[slots] = 0.0
        got = run_recurrence(ops, case, inputs, gates_in, portions, state, slots)
        for r, b in enumerate(want):
            error = (got[r] - b).abs().max() / max(1.0, float(b.abs().max()))
            assert error < tolerance, f"request {r} portions {portions[r]}: {error}"
    unused = [slot for slot in range(7) if slot not in [(r * 3 + t) % 7 for t in range(4) for r in range(5)]]
    assert all((state[slot] == 5.0).all() for slot in unused)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_recurrence_over_a_long_prompt(ops, dtype):
    """Thousands of tokens (longer chunks, many a channel) beside a short request, and the same in two
    portions of which the second is long again."""
    case = recurrence_case(16, 2, dtype, 1, lam=-5.0)
    generator = torch.Generator().manual_seed(2)
    inputs, gates_in = ([torch.randn(n, 16, generator=generator).to(dtype) for n in (4500, 40)] for _ in range(2))
    want = [plain_recurrence(x, y, case) for x, y in zip(inputs, gates_in)]
    for portions in (((5000,), (5000,)), ((201, 5000), (39, 1)), ((4300, 200), (40,))):
        state = torch.zeros(2, 16, device=DEVICE)
        got = run_recurrence(ops, case, inputs, gates_in, portions, state, [1, 0])
        for r, b in enumerate(want):
            error = (got[r] - b).abs().max() / max(1.0, float(b.abs().max()))
            assert error < (2e-4 if dtype == torch.float32 else 0.03), f"request {r} portions {portions[r]}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_channels_that_keep_and_channels_that_forget(ops, dtype):
    """Decays within a millionth of 1 (where 1 - a^2 taken as a difference would be noise) and decays
    that underflow: what the third token brought still moves some channels 1100 tokens later, by
    decoding and in a prompt of several chunks."""
    width = 64
    case = recurrence_case(width, 4, dtype, 3)
    for name in ("ra", "ri", "ra_b"):
        case[name].zero_()
    case["ri_b"].fill_(3.0)
    case["lam"] = torch.cat([torch.full((32,), -13.0), torch.full((16,), -8.0), torch.full((16,), 30.0)])
    generator = torch.Generator().manual_seed(9)
    u = 0.3 * torch.randn(1100, width, generator=generator)
    u[2] = 60.0
    u, y = u.to(dtype), (1.0 + torch.randn(1100, width, generator=generator)).to(dtype)
    want = plain_recurrence(u, y, case)
    changed = u.clone()
    changed[2] *= -1.0
    moved = (plain_recurrence(changed, y, case) - want)[-20:].abs().amax(0)
    assert moved[:32].min() > 0.02 and moved[48:].max() == 0
    for portions in (((2000,),), ((333, 2, 200, 1),), ((1,),)):
        state = torch.zeros(1, width, device=DEVICE)
        (got,) = run_recurrence(ops, case, [u], [y], portions, state, [0])
        assert torch.isfinite(got).all()
        error = ((got - want).abs() / torch.clamp(want.abs(), min=0.1))
        assert error.max() < (2e-3 if dtype == torch.float32 else 0.03), str(portions)
        # (a decay that close to 1 is off by half a unit of 2^-24 in 32-bit, and so token after token)
        bound = 1e-4 if dtype == torch.float32 else 0.02
        assert ((got - want).abs() < bound * torch.clamp(want.abs(), min=1.0)).all(), str(portions)


# ------------------------------------------------------------------ clamped experts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, hidden, width, boundary, limits", [
    (1, 64, 96, 60, (0.8, 1.4)), (7, 128, 40, 40, (1.0, 9.0)), (16, 256, 304, 200, (0.5, 2.0)), (40, 72, 50, 13, (1.1, 0.6)),
    (300, 128, 256, 256, (0.9, 0.9)), (513, 256, 1024, 0, (5.0, 0.7)), (140, 64, 136, 64, (0.7, 1.5)), (3, 20, 30, 17, (0.7, 1.5))])
def test_clamped_gates(ops, dtype, rows, hidden, width, boundary, limits):
    """Every way that the product takes (few rows, many, with two limits and with one), with values on
    both sides of the limits."""
    generator = torch.Generator().manual_seed(rows)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    x, w = draw(rows, hidden).to(dtype), (1.5 * draw(2 * width, hidden) / hidden ** 0.5).to(dtype)
    got = ops.linear_gated(on(x), on(w), "clamped", limits=(*limits, boundary)).cpu().double()
    ops.check_errors()
    both = x.double() @ w.double().T
    limit = torch.where(torch.arange(width) < boundary, limits[0], limits[1]).double()
    g, u = torch.minimum(both[:, :width], limit), both[:, width:]
    u = torch.maximum(torch.minimum(u, limit), -limit)
    assert (both[:, :width] > limit).any() and (both[:, width:] < -limit).any() or limits[0] > 4 or limits[1] > 4
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    assert (got - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.04)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden, width, experts, top, shared", [
    (64, 40, 9, 2, (48, 1.4)), (96, 24, 8, 2, None), (256, 136, 16, 4, (264, 0.5)), (72, 20, 6, 6, (12, 2.0)),
    (128, 304, 4, 1, (304, 0.9)), (52, 20, 5, 1, None), (40, 8, 1, 1, (16, 0.6))])
def test_clamped_experts(dtype, hidden, width, experts, top, shared):
    """One token, a few, enough to be sorted by expert (grouped products), also where an expert gets
    more than a tile of them; the shared expert has a limit of its own."""
    from mlx_one_b200.architectures.zinizen import _feed_forward
    from mlx_one_b200.config.zinizen import RoutedFeedForward
    from mlx_one_b200.parts import FEED_FORWARDS

    generator = torch.Generator().manual_seed(width)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    m = {"kind": "moe", "expert": {"ff": width, "limit": 0.9},
         "router": {"experts": experts, "top": top, "scale": 1.7}}
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    spec = _feed_forward(RoutedFeedForward.from_dict(m, ""), hidden)
    cls = FEED_FORWARDS.get("routed")
    w = {}
    for name, want in cls.tensors(spec).items():
        values = draw(*want.shape)
        if name == "correction":
            values = 0.1 * values
        else:
            values = (3.0 if name == "router" else 1.5) * values / want.shape[1] ** 0.5
        w[name] = values.to(dtype)
    part = cls(spec, {name: on(t) for name, t in w.items()}, runtime(dtype))
    wide = {name: t.double() for name, t in w.items()}
    for tokens, shift in ((1, 0.0), (2, 0.0), (7, 0.0), (40, 0.0), (200, 0.0), (450, 2.0)):
        x = draw(tokens, hidden)
        x = (x + shift * wide["router"][0].float() / wide["router"][0].float().norm()).to(dtype)
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


def test_the_stream_after_every_layer(folders, models):
    for name in ("Z1", "Z2", "Z4"):
        config, _, page = CONFIGS[name]
        runner, cache = engine(folders[name], torch.float32, page, 64)
        (tokens,) = prompts(config["vocab"], (19,), seed=2)
        seen = []

        def observe(place, residual, update):
            if place >= 0:
                seen.append(update.applied(residual))

        runner.model.observer = observe
        replay(runner, cache, [([("r", tokens)], ["r"])])
        runner.model.observer = None
        states = []
        models[name].logits(tokens, states)
        assert len(seen) == len(states) == len(config["layers"])
        for place, (got, want) in enumerate(zip(seen, states)):
            # (a step's rows may be padded to a shape that is replayed)
            got = got[:len(tokens)].cpu().double()
            assert (got - want).abs().max() < 5e-4, f"{name} after layer {place}"


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
@pytest.mark.parametrize("name", ["Z1", "Z4"])
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
def test_many_requests_decode_side_by_side(folders, models, dtype):
    """Twenty requests, more than the recurrence's single-token kernel takes."""
    config, _, page = CONFIGS["Z4"]
    requests = dict(enumerate(prompts(config["vocab"], [5 + i for i in range(20)], seed=11)))
    runner, cache = engine(folders["Z4"], dtype, page, 20 * 64, max_requests=20)
    steps = [([(key, tokens[:3]) for key, tokens in requests.items()], [])]
    for i in range(3, 24):
        live = [(key, [tokens[i]]) for key, tokens in requests.items() if i < len(tokens)]
        if live:
            steps.append((live, [key for key, tokens in requests.items() if i == len(tokens) - 1]))
    got = replay(runner, cache, steps)
    for key, tokens in requests.items():
        assert_close(got[key], models["Z4"].logits(tokens), dtype, f"request {key}")
    assert not cache.requests()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_far_keys(tmp_path, dtype):
    """A prompt in portions that cut pages and chunks, then 260 tokens decoded one by one; the third
    token still moves the last logits (the plain model says by how much)."""
    config = {"architecture": "Zinizen", "vocab": 200, "width": 64, "norm": {"eps": 1e-5},
              "embedding": bigram(50, 3, 7),
              "layers": [attention(8, 4, 16, 16, 0.3, dense(128), 6.0, (0.3, 100), True),
                         rglru(64, 4, 4, dense(128)), latent(2, 24, 16, 40, 56, 40, 0.25, None, base=50000.0),
                         attention(8, 4, 16, 16, 0.3, None, 6.0, (0.3, 100), True), rglru(96, 2, 3, dense(96))]}
    folder = make_model_dir("Z1", tmp_path, config)
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

    for name, dtype in (("Z1", "float32"), ("Z4", "float32"), ("Z2", "bfloat16")):
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
    folder = folders["Z4"]
    greedy = subprocess.run([sys.executable, str(root / "bin" / "mlx-one"), "generate", str(folder),
                             "5 17 3 200", "--token-ids", "--max-tokens", "6", "--dtype", "float32"],
                            capture_output=True, text=True, timeout=600)
    assert greedy.returncode == 0, greedy.stderr
    assert [int(t) for t in greedy.stdout.split()] == models["Z4"].greedy([5, 17, 3, 200], 6)

    vocab = CONFIGS["Z4"][0]["vocab"]
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
    wa, wb, wc = (models["Z4"].logits(t) for t in (a, b, c))
    close = lambda got, want: (got - want).abs().max() < 5e-4
    assert close(read(0, 3), torch.stack([wa[0], wa[7], wb[8]]))
    assert close(read(2, 2), torch.stack([wa[20], wc[1]]))
    assert close(read(3, 1), wc[29:30])

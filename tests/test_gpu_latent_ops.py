"""Operators around latent attention, output norms, gated feed-forwards and mixtures of experts, each alone,
against float64 statements (kikepel_oracle.py): odd and unequal sizes, both activation types, every kernel behind an
operator, keys at every kind of edge."""
from __future__ import annotations

import ctypes

import numpy as np
import pytest

import kikepel_oracle as oracle
from gpu_util import stream

pytestmark = pytest.mark.gpu
TYPES = pytest.mark.parametrize("float32", [0, 1], ids=["bf16", "f32"])


def cuda(values, dtype=None):
    import torch

    tensor = torch.from_numpy(np.ascontiguousarray(values))
    return tensor.to("cuda", dtype or tensor.dtype)


def activation(values, float32):
    """Device tensor in the activation type, and the float64 values it holds."""
    import torch

    tensor = cuda(np.asarray(values, np.float32), torch.float32 if float32 else torch.bfloat16)
    return tensor, tensor.double().cpu().numpy()


def empty(shape, float32):
    import torch

    return torch.full(shape, float("nan"), dtype=torch.float32 if float32 else torch.bfloat16, device="cuda")


def integers(shape):
    import torch

    return torch.full(shape, -1, dtype=torch.int32, device="cuda")


def call(ops, name, arguments):
    ops.call(name, ctypes.addressof(arguments), stream())
    ops.call("check_async_errors", stream())


def assert_near(actual, expected, float32, factor=1.0):
    actual = actual.double().cpu().numpy() if hasattr(actual, "cpu") else actual
    bound = (2e-5 if float32 else 1.2e-2) * factor
    scale = np.sqrt(np.mean(expected * expected)) + 1e-30
    worst = np.max(np.abs(actual - expected) / (np.abs(expected) + scale))
    assert np.isfinite(actual).all() and worst < bound, (worst, bound)


# ---------------------------------------------------------------- norms and embedding
@TYPES
@pytest.mark.parametrize("input32", [0, 1])
@pytest.mark.parametrize("width", [1, 8, 77, 1536, 2056, 4104, 8200, 16392])
def test_layer_norm(pkg, ops, float32, input32, width):
    rng = np.random.default_rng(width)
    rows, parts, eps = 5, 3, 1e-3
    x, xv = activation(rng.normal(0.4, 0.3, (rows * parts + 7, width)), input32)
    gain, residual = rng.uniform(0.5, 1.5, width).astype(np.float32), rng.normal(0, 1, (rows, width)).astype(np.float32)
    slots = rng.permutation(rows * parts + 7)[:rows * parts].astype(np.int32).reshape(rows, parts)
    dg, ds = cuda(gain), cuda(slots)
    common = dict(input=x.data_ptr(), gain=dg.data_ptr(), rows=rows, width=width, epsilon=eps, input_float32=input32,
                  output_float32=float32)
    for use_slots in (False, True):
        order = slots if use_slots else np.arange(rows * parts).reshape(rows, parts)
        normed = oracle.layer_norm(xv[order].sum(axis=1), gain.astype(np.float64), eps)
        out = empty((rows, width), float32)
        call(ops, "layer_norm", pkg.LayerNorm(**common, parts=parts, slots=ds.data_ptr() if use_slots else None,
                                              output=out.data_ptr()))
        assert_near(out, normed, float32, factor=5.0 if width == 1 else 2.0)
    dr, copy = cuda(residual), empty((rows, width), float32)
    call(ops, "layer_norm", pkg.LayerNorm(**common, parts=1, residual=dr.data_ptr(), output=copy.data_ptr()))
    expected = residual + oracle.layer_norm(xv[:rows], gain.astype(np.float64), eps)
    assert_near(dr, expected, 1)                                     # the stream itself is F32 in both types
    assert_near(copy, dr.double().cpu().numpy(), float32)
    dr = cuda(residual)
    call(ops, "layer_norm", pkg.LayerNorm(**common, parts=1, residual=dr.data_ptr()))
    assert_near(dr, expected, 1)


def test_layer_norm_of_a_far_mean(pkg, ops):
    """The variance comes from the deviations: a mean a thousand times the spread does not drown it."""
    rng = np.random.default_rng(0)
    x = (1000.0 + rng.normal(0, 1, (3, 600))).astype(np.float32)
    dx, dg, out = cuda(x), cuda(np.ones(600, np.float32)), empty((3, 600), 1)
    call(ops, "layer_norm", pkg.LayerNorm(input=dx.data_ptr(), gain=dg.data_ptr(), output=out.data_ptr(), parts=1, rows=3,
                                          width=600, epsilon=1e-6, input_float32=1, output_float32=1))
    assert_near(out, oracle.layer_norm(x.astype(np.float64), np.ones(600), 1e-6), 1, factor=20.0)


@TYPES
@pytest.mark.parametrize("width", [48, 51, 4104])
def test_embedding_rows(ops, float32, width):
    rng = np.random.default_rng(width)
    table, tv = activation(rng.normal(0, 1, (30, width)), 0)
    tokens = cuda(np.array([3, 29, 0, 3, 30], np.int32))             # the last id is outside the vocabulary
    out, copy = empty((5, width), 1), empty((5, width), float32)
    ops.call("embed_rows", tokens.data_ptr(), table.data_ptr(), 4, width, 30, out.data_ptr(), copy.data_ptr(), float32, stream())
    ops.call("check_async_errors", stream())
    assert (out[:4].double().cpu().numpy() == tv[[3, 29, 0, 3]]).all() and bool((copy[:4].float() == out[:4]).all())
    ops.call("embed_rows", tokens.data_ptr(), table.data_ptr(), 5, width, 30, out.data_ptr(), None, float32, stream())
    assert ops.status("check_async_errors", stream()) == 2 and not out[4].any()


@TYPES
@pytest.mark.parametrize("query_rank, latent_rank", [(40, 72), (1, 1), (33, 2100), (3000, 512)])
def test_latent_norms(pkg, ops, float32, query_rank, latent_rank):
    rng = np.random.default_rng(query_rank)
    rows, position, capacity, column = 5, 11, 18, (query_rank + 7) // 8 * 8
    p, pv = activation(rng.normal(0, 0.1, (rows, column + latent_rank + 3)), float32)
    qg, cg = rng.uniform(0.5, 1.5, query_rank).astype(np.float32), rng.uniform(0.5, 1.5, latent_rank).astype(np.float32)
    dq, dc, query, cache = cuda(qg), cuda(cg), empty((rows, query_rank), float32), empty((capacity, latent_rank), float32)
    call(ops, "latent_norm_append", pkg.LatentNorm(
        projection=p.data_ptr(), query_gain=dq.data_ptr(), latent_gain=dc.data_ptr(), query_latent=query.data_ptr(),
        cache=cache.data_ptr(), stride=column + latent_rank + 3, latent_column=column, rows=rows, position=position,
        capacity=capacity, query_rank=query_rank, latent_rank=latent_rank, epsilon=1e-3, float32=float32))
    assert_near(query, oracle.rms(pv[:, :query_rank], 1e-3) * qg, float32)
    assert_near(cache[position:position + rows], oracle.rms(pv[:, column:column + latent_rank], 1e-3) * cg, float32)
    kept = cache.float().cpu().numpy()
    assert np.isnan(kept[:position]).all() and np.isnan(kept[position + rows:]).all()


# ---------------------------------------------------------------- projections
GATES = {3: lambda a, b, limit: np.maximum(a, 0.0) * b,
         4: lambda a, b, limit: np.minimum(a, limit) * oracle.sigmoid(1.702 * np.minimum(a, limit)) * (np.clip(b, -limit, limit) + 1.0)}


def interleave(gate, up):
    """Blocks of 128 gate rows and 128 up rows in turn."""
    blocks = [m.reshape(-1, 128, *m.shape[1:]) for m in (gate, up)]
    return np.stack(blocks, axis=1).reshape(-1, *gate.shape[1:])


@pytest.mark.parametrize("gate", [3, 4])
@pytest.mark.parametrize("rows", [1, 3, 8, 16, 33, 64, 100, 129, 600])
@pytest.mark.parametrize("inner, columns", [(64, 128), (200, 384), (1024, 256)])
def test_gated_projections(pkg, ops, gate, rows, inner, columns):
    rng = np.random.default_rng(rows + inner)
    x, xv = activation(rng.normal(0, 1, (rows, inner)), 0)
    (_, a), (_, b) = (activation(rng.normal(0, inner ** -0.5, (columns, inner)), 0) for _ in range(2))
    w, _ = activation(interleave(a, b), 0)
    bias_a, bias_b = rng.normal(0, 1, (2, columns)).astype(np.float32)
    db = cuda(interleave(bias_a, bias_b))
    work = empty((1 << 22,), 1)
    biased = gate == 3
    expected = GATES[gate](xv @ a.T + biased * bias_a, xv @ b.T + biased * bias_b, 0.9)
    for workspace in (0, work.numel() * 4):
        out = empty((rows, columns), 0)
        call(ops, "projection", pkg.Projection(
            input=x.data_ptr(), weight=w.data_ptr(), bias=db.data_ptr() if biased else None, output=out.data_ptr(), rows=rows,
            in_features=inner, out_features=2 * columns, alpha=1.0, gate=gate, gate_limit=0.9,
            split_workspace=work.data_ptr() if workspace else None, split_workspace_bytes=workspace))
        assert_near(out, expected, 0)


@TYPES
@pytest.mark.parametrize("gate", [3, 4])
def test_gated_activation(ops, float32, gate):
    rng = np.random.default_rng(gate)
    a, b = rng.normal(0, 2, (2, 300, 384)).astype(np.float32)
    a[0, 0], a[0, 1], a[0, 2] = -200.0, 200.0, 0.0
    products = cuda(np.ascontiguousarray(interleave(a.T, b.T).T))
    out, count = empty((300, 384), float32), cuda(np.array([2], np.int32))
    ops.call("gated_activation", products.data_ptr(), gate, 1.3, 300, 384, out.data_ptr(), float32, None, 0, stream())
    expected = GATES[gate](a.astype(np.float64), b.astype(np.float64), 1.3)
    assert_near(out, expected, float32)
    out.fill_(float("nan"))
    ops.call("gated_activation", products.data_ptr(), gate, 1.3, 300, 384, out.data_ptr(), float32, count.data_ptr(), 64, stream())
    assert_near(out[:128], expected[:128], float32)
    assert bool(out[128:].isnan().all())


@pytest.mark.parametrize("rows", [1, 5, 16, 40, 100, 300, 600])
@pytest.mark.parametrize("inner, outer", [(72, 300), (64, 1030), (51, 37)])
def test_capped_logits(pkg, ops, rows, inner, outer):
    rng = np.random.default_rng(rows * outer)
    x, xv = activation(rng.normal(0, 1, (rows, inner)), 0)
    w, wv = activation(rng.normal(0, 1, (outer, inner)), 0)
    exact = cuda(rng.normal(0, 1, (rows, inner)).astype(np.float32))
    work = empty((1 << 22,), 1)
    for scale, cap in ((2.5, 11.0), (0.01, 50.0), (40.0, 3.0)):
        arguments = dict(weight=w.data_ptr(), rows=rows, in_features=inner, out_features=outer, alpha=scale, softcap=cap,
                         f32_result=1, row_fanout=1)
        for float32, source, values in ((0, x, xv), (1, exact, exact.double().cpu().numpy()), (2, x, xv)):
            out = empty((rows, outer), 1)
            call(ops, "projection", pkg.Projection(input=source.data_ptr(), output=out.data_ptr(), float32=float32,
                                                   split_workspace=work.data_ptr(), split_workspace_bytes=work.numel() * 4,
                                                   **arguments))
            expected = oracle.capped_logits(values, wv, scale, cap)
            assert_near(out, expected, 1, factor=5.0)


# ---------------------------------------------------------------- mixture of experts
def expected_route(logits, top):
    order = np.argsort(-logits, axis=1, kind="stable")[:, :top]
    return order, oracle.sigmoid(np.take_along_axis(logits, order, axis=1))


@TYPES
@pytest.mark.parametrize("rows, width, experts, top", [(1, 64, 5, 1), (3, 51, 12, 3), (8, 2048, 64, 8), (2, 72, 1, 1), (5, 40, 300, 300),
                                                      (1, 96, 1024, 2)])
def test_router_with_its_own_products(pkg, ops, float32, rows, width, experts, top):
    rng = np.random.default_rng(experts)
    x, xv = activation(rng.normal(0, 1, (rows, width)), float32)
    router, rv = activation(rng.normal(0, width ** -0.5, (experts, width)), 0)
    expert, score = integers((rows, top)), empty((rows, top), 1)
    call(ops, "route_rows", pkg.Route(input=x.data_ptr(), router=router.data_ptr(), rows=rows, width=width, experts=experts,
                                      top=top, expert=expert.data_ptr(), score=score.data_ptr(), float32=float32))
    logits = xv @ rv.T
    chosen, scores = expected_route(logits, top)
    assert_near(score, scores, 1)
    mine = np.take_along_axis(logits, expert.cpu().numpy().astype(np.int64), axis=1)
    assert np.abs(mine - np.take_along_axis(logits, chosen, axis=1)).max() < 1e-5       # equal up to near ties
    assert all(len(set(row)) == top for row in expert.cpu().numpy().tolist())


@pytest.mark.parametrize("rows, experts, top, stride", [(1, 3, 2, 64), (700, 40, 4, 64), (300, 130, 9, 192), (33, 900, 1, 960)])
def test_router_choice_counts_and_ranks(pkg, ops, rows, experts, top, stride):
    rng = np.random.default_rng(rows)
    logits = rng.normal(0, 2, (rows, stride)).astype(np.float32)
    logits[:, experts:] = 100.0                                       # padding columns are no experts
    logits[0, :experts] = 0.25                                        # ties go to the lower index
    dl, expert, score = cuda(logits), integers((rows, top)), empty((rows, top), 1)
    counts, rank = integers((experts,)), integers((rows, top))
    call(ops, "route_rows", pkg.Route(logits=dl.data_ptr(), logit_stride=stride, rows=rows, experts=experts, top=top,
                                      expert=expert.data_ptr(), score=score.data_ptr(), counts=counts.data_ptr(),
                                      rank=rank.data_ptr()))
    chosen, scores = expected_route(logits[:, :experts].astype(np.float64), top)
    assert (expert.cpu().numpy() == chosen).all()
    assert_near(score, scores, 1)
    assert (counts.cpu().numpy() == np.bincount(chosen.ravel(), minlength=experts)).all()
    ranks = rank.cpu().numpy()
    for e in range(experts):
        assert sorted(ranks[chosen == e]) == list(range((chosen == e).sum()))


def grouped(pkg, ops, x, chosen, scores, experts, tile_rows, float32):
    """Rows in their experts' tiles through the library: (rows, slot scores, slot, tile_group, tile_count, capacity)."""
    rows, width = x.shape
    top = chosen.shape[1]
    counts = np.bincount(chosen.ravel(), minlength=experts).astype(np.int32)
    rank = np.zeros(chosen.shape, np.int32)
    for e in range(experts):
        rank[chosen == e] = np.arange(counts[e])
    tiles = ops.lib.evo_b200_grouped_tiles(rows, top, experts, tile_rows)
    capacity = tiles * tile_rows
    keep = [cuda(v) for v in (chosen.astype(np.int32), rank, counts, scores.astype(np.float32))]
    out, slot_score = empty((capacity, width), float32), empty((capacity,), 1)
    slot, tile_group, tile_count = integers((rows, top)), integers((tiles,)), integers((1,))
    call(ops, "group_rows", pkg.GroupRows(
        input=x.data_ptr(), expert=keep[0].data_ptr(), rank=keep[1].data_ptr(), counts=keep[2].data_ptr(),
        score=keep[3].data_ptr(), grouped=out.data_ptr(), slot_score=slot_score.data_ptr(), slot=slot.data_ptr(),
        tile_group=tile_group.data_ptr(), tile_count=tile_count.data_ptr(), rows=rows, width=width, experts=experts, top=top,
        tile_rows=tile_rows, float32=float32))
    used = -(-counts // tile_rows)
    assert int(tile_count[0]) == used.sum() <= tiles
    assert (tile_group.cpu().numpy()[:used.sum()] == np.repeat(np.arange(experts), used)).all()
    return out, slot_score, slot, tile_group, tile_count, capacity


@TYPES
@pytest.mark.parametrize("rows, width, experts, top, tile_rows", [(9, 51, 7, 2, 128), (500, 72, 5, 3, 128), (700, 64, 3, 1, 256),
                                                                 (40, 8, 130, 4, 128)])
def test_rows_are_grouped_by_expert(pkg, ops, float32, rows, width, experts, top, tile_rows):
    rng = np.random.default_rng(rows)
    x, _ = activation(rng.normal(0, 1, (rows, width)), float32)
    chosen = np.stack([rng.permutation(experts)[:top] for _ in range(rows)])
    scores = rng.uniform(0, 1, chosen.shape)
    out, slot_score, slot, _, _, _ = grouped(pkg, ops, x, chosen, scores, experts, tile_rows, float32)
    at = slot.cpu().numpy()
    assert len(set(at.ravel())) == rows * top
    for k in range(top):
        assert bool((out[at[:, k]] == x).all())
        assert np.allclose(slot_score.cpu().numpy()[at[:, k]], scores[:, k])


@pytest.mark.parametrize("tile_rows", [128, 256])
@pytest.mark.parametrize("rows, width, inner, experts, top", [(50, 72, 128, 6, 2), (700, 264, 256, 5, 2), (1500, 320, 384, 2, 1), (33, 64, 128, 40, 3)])
def test_experts_in_tiles(pkg, ops, tile_rows, rows, width, inner, experts, top):
    """Regrouped rows through gated and plain grouped projections and the norm that sums a row's experts, against
    the same thing row by row; skewed loads, experts that nobody chose."""
    rng = np.random.default_rng(rows)
    if tile_rows == 256 and width < 256:
        pytest.skip("CTA pairs work on 256 output columns")
    x, xv = activation(rng.normal(0, 1, (rows, width)), 0)
    popularity = rng.normal(0, 1, (rows, experts)) + np.linspace(2, -2, experts)
    popularity[:, 1 if experts > 2 else 0] = -50.0 if experts > top + 1 else 0.0
    chosen, scores = expected_route(popularity, top)
    (_, a), (_, b) = (activation(rng.normal(0, width ** -0.5, (experts, inner, width)), 0) for _ in range(2))
    up, _ = activation(np.concatenate([interleave(a[e], b[e]) for e in range(experts)]), 0)
    down, dv = activation(rng.normal(0, inner ** -0.5, (experts, width, inner)), 0)
    source, slot_score, slot, tile_group, tile_count, capacity = grouped(pkg, ops, x, chosen, scores, experts, tile_rows, 0)
    tiles = dict(tile_group=tile_group.data_ptr(), tile_count=tile_count.data_ptr(), tile_rows=tile_rows, groups=experts,
                 row_fanout=1, rows=capacity)
    gated, result = empty((capacity, inner), 0), empty((capacity, width), 0)
    call(ops, "projection", pkg.Projection(input=source.data_ptr(), weight=up.data_ptr(), output=gated.data_ptr(), in_features=width,
                                           out_features=2 * inner, alpha=1.0, gate=4, gate_limit=0.7,
                                           row_scale=slot_score.data_ptr(), **tiles))
    call(ops, "projection", pkg.Projection(input=gated.data_ptr(), weight=down.data_ptr(), output=result.data_ptr(), in_features=inner,
                                           out_features=width, alpha=1.0, **tiles))
    residual, gain = cuda(np.zeros((rows, width), np.float32)), cuda(np.ones(width, np.float32))
    call(ops, "layer_norm", pkg.LayerNorm(input=result.data_ptr(), slots=slot.data_ptr(), gain=gain.data_ptr(), parts=top, rows=rows,
                                          residual=residual.data_ptr(), width=width, epsilon=1e-6, input_float32=0))
    scores = scores.astype(np.float32).astype(np.float64)
    summed, middle = np.zeros((rows, width)), np.zeros((rows, top, inner))
    for r in range(rows):
        for k, e in enumerate(chosen[r]):
            scaled = scores[r, k] * xv[r]
            middle[r, k] = GATES[4](a[e] @ scaled, b[e] @ scaled, 0.7)
            summed[r] += dv[e] @ middle[r, k]
    at = slot.cpu().numpy()
    assert_near(gated[at], middle, 0)
    assert_near(residual, oracle.layer_norm(summed, np.ones(width), 1e-6), 0, factor=2.0)
    # the kernels of the F32 profile on the same tiles
    for float32 in (2, 1):
        exact = source if float32 == 2 else cuda(source.float().cpu().numpy())
        products = empty((capacity, 2 * inner), 1)
        call(ops, "projection", pkg.Projection(input=exact.data_ptr(), weight=up.data_ptr(), output=products.data_ptr(), alpha=1.0,
                                               in_features=width, out_features=2 * inner, float32=float32, f32_result=1,
                                               row_scale=slot_score.data_ptr(), **tiles))
        ops.call("gated_activation", products.data_ptr(), 4, 0.7, capacity, inner, gated.data_ptr(), 0, tile_count.data_ptr(),
                 tile_rows, stream())
        assert_near(gated[at], middle, 0)


@pytest.mark.parametrize("rows, top, width, inner", [(1, 1, 72, 128), (1, 4, 1024, 384), (7, 3, 64, 256), (8, 2, 200, 128)])
def test_experts_pair_by_pair(pkg, ops, rows, top, width, inner):
    rng = np.random.default_rng(rows + width)
    experts = 9
    x, xv = activation(rng.normal(0, 1, (rows, width)), 0)
    chosen, scores = expected_route(rng.normal(0, 1, (rows, experts)), top)
    (_, a), (_, b) = (activation(rng.normal(0, width ** -0.5, (experts, inner, width)), 0) for _ in range(2))
    up, _ = activation(np.concatenate([interleave(a[e], b[e]) for e in range(experts)]), 0)
    down, dv = activation(rng.normal(0, inner ** -0.5, (experts, width, inner)), 0)
    group, score = cuda(chosen.astype(np.int32)), cuda(scores.astype(np.float32))
    pairs = rows * top
    gated, result = empty((pairs, inner), 0), empty((pairs, width), 0)
    call(ops, "projection", pkg.Projection(input=x.data_ptr(), weight=up.data_ptr(), output=gated.data_ptr(), rows=pairs,
                                           in_features=width, out_features=2 * inner, alpha=1.0, gate=4, gate_limit=0.7,
                                           row_scale=score.data_ptr(), row_group=group.data_ptr(), row_fanout=top, groups=experts))
    middle = np.array([[GATES[4](a[e] @ (s * xv[r]), b[e] @ (s * xv[r]), 0.7) for e, s in zip(chosen[r], scores[r])]
                       for r in range(rows)]).reshape(pairs, inner)
    assert_near(gated, middle, 0)
    call(ops, "projection", pkg.Projection(input=gated.data_ptr(), weight=down.data_ptr(), output=result.data_ptr(), rows=pairs,
                                           in_features=inner, out_features=width, alpha=1.0, row_group=group.data_ptr(),
                                           row_fanout=1, groups=experts))
    expected = np.stack([dv[e] @ m for e, m in zip(chosen.ravel(), gated.double().cpu().numpy())])
    assert_near(result, expected, 0)
    exact, products = cuda(xv.astype(np.float32)), empty((pairs, 2 * inner), 1)
    call(ops, "projection", pkg.Projection(input=exact.data_ptr(), weight=up.data_ptr(), output=products.data_ptr(), rows=pairs,
                                           in_features=width, out_features=2 * inner, alpha=1.0, row_scale=score.data_ptr(), float32=1,
                                           f32_result=1, row_group=group.data_ptr(), row_fanout=top, groups=experts))
    precise = empty((pairs, inner), 1)
    ops.call("gated_activation", products.data_ptr(), 4, 0.7, pairs, inner, precise.data_ptr(), 1, None, 0, stream())
    assert_near(precise, middle, 1)


def test_grouped_refusals(pkg, ops):
    x, w, out, group = empty((8, 51), 0), empty((4 * 256, 51), 0), empty((8, 128), 0), integers((8,))
    common = dict(input=x.data_ptr(), weight=w.data_ptr(), output=out.data_ptr(), rows=8, in_features=51, out_features=256,
                  alpha=1.0, groups=4, row_fanout=1, tile_rows=128)
    for grouping in (dict(row_group=group.data_ptr()), dict(tile_group=group.data_ptr(), tile_count=group.data_ptr())):
        with pytest.raises(pkg.OpsError) as error:                    # no tensor map or vector load at this width
            call(ops, "projection", pkg.Projection(**common, **grouping))
        assert error.value.code == 5
    with pytest.raises(pkg.OpsError) as error:
        call(ops, "projection", pkg.Projection(input=x.data_ptr(), weight=w.data_ptr(), output=out.data_ptr(), rows=8, in_features=51,
                                               out_features=256, alpha=1.0, gate=4, f32_result=1))
    assert error.value.code == 2


# ---------------------------------------------------------------- attention
def last_rows(q, k, v, *, scale, window, sink):
    """oracle.attention of the last len(q) rows alone."""
    position = len(k) - len(q)
    out = np.zeros((*q.shape[:2], v.shape[2]))
    for r in range(len(q)):
        seen = oracle.visible_keys(position + r, window)
        for h in range(q.shape[1]):
            g = h // (q.shape[1] // k.shape[1])
            out[r, h] = oracle.softmax((k[seen, g] @ q[r, h]) * scale, None if sink is None else float(sink[h])) @ v[seen, g]
    return out


def attention_case(pkg, ops, *, rows, position, heads, kv_heads, dim, vdim, window, kernel, float32=0, sinks=True, seed=0,
                   edit=None, sink_range=(-2.0, 4.0)):
    """Plain softmax in a window with learned sinks; returns (output, expected [rows, heads, vdim])."""
    rng = np.random.default_rng(seed)
    total, capacity = position + rows, position + rows + 5
    q, k, v = (rng.normal(0, 1, shape) for shape in ((rows, heads, dim), (capacity, kv_heads, dim), (capacity, kv_heads, vdim)))
    if edit is not None:
        edit(q, k, v)
    k[total:], v[total:] = 1e4, 1e4                                 # what lies behind the last key is never read
    (dq, q), (dk, k), (dv, v) = (activation(x, float32) for x in (q, k, v))
    sink = rng.uniform(*sink_range, heads).astype(np.float32)
    ds, out = cuda(sink), empty((rows, heads, vdim), float32)
    call(ops, "window_attention", pkg.WindowAttention(
        query=dq.data_ptr(), key_cache=dk.data_ptr(), value_cache=dv.data_ptr(), output=out.data_ptr(), rows=rows, position=position,
        capacity=capacity, heads=heads, kv_heads=kv_heads, dim=dim, value_dim=vdim, window=window, scale=dim ** -0.5,
        sink=int(sinks), sink_logit=ds.data_ptr(), float32=float32, kernel=kernel))
    return out, last_rows(q, k[:total], v[:total], scale=dim ** -0.5, window=window, sink=sink if sinks else None)


ROW, TILE, TENSOR = 1, 2, 3
KERNELS = pytest.mark.parametrize("kernel", [ROW, TILE, TENSOR], ids=["row", "tile", "tensor"])


@KERNELS
@pytest.mark.parametrize("sinks", [True, False])
def test_attention_with_learned_sinks(pkg, ops, kernel, sinks):
    for rows, position, window in ((1, 0, 5), (70, 40, 33), (140, 0, 500), (65, 300, 64)):
        out, expected = attention_case(pkg, ops, rows=rows, position=position, heads=3, kv_heads=3, dim=64, vdim=72, window=window,
                                       kernel=kernel, sinks=sinks, seed=rows)
        assert_near(out, expected, 0, factor=2.0)


@KERNELS
@pytest.mark.parametrize("low, high", [(-300.0, -200.0), (30.0, 60.0), (200.0, 400.0)])
def test_extreme_sinks(pkg, ops, kernel, low, high):
    """A sink far below every score changes nothing, one far above takes everything."""
    out, expected = attention_case(pkg, ops, rows=66, position=10, heads=2, kv_heads=1, dim=64, vdim=64, window=20, kernel=kernel,
                                   sink_range=(low, high))
    if high < 0:
        assert_near(out, expected, 0, factor=2.0)
    else:
        assert np.isfinite(out.float().cpu().numpy()).all() and np.abs(out.float().cpu().numpy()).max() < 1e-6


@TYPES
@pytest.mark.parametrize("rank", [260, 512, 604, 1024])
def test_wide_heads_in_the_row_kernel(pkg, ops, float32, rank):
    for rows, position, window in ((1, 0, 9), (1, 130, 40), (8, 60, 31), (3, 9, 300)):
        out, expected = attention_case(pkg, ops, rows=rows, position=position, heads=5, kv_heads=1, dim=rank, vdim=rank, window=window,
                                       kernel=0, float32=float32, seed=rank + rows)
        assert_near(out, expected, float32)


@pytest.mark.parametrize("kernel, dim", [(ROW, 64), (TILE, 64), (TENSOR, 64), (ROW, 520), (TILE, 32)])
@pytest.mark.parametrize("key_at", ["oldest in the window", "just outside", "own", "next"])
def test_one_key_stands_out(pkg, ops, kernel, dim, key_at):
    """One key that every query scores far above the rest, at the edges of what a query sees: its value dominates
    exactly where it is visible."""
    rows, position, window = (140, 200, 50) if kernel != ROW else (70, 200, 50)
    target = {"oldest in the window": position + 60 - window + 1, "just outside": position + 60 - window, "own": position + 60,
              "next": position + 61}[key_at]

    def plant(q, k, v):
        q[..., 0], k[..., 0] = 4.0, 0.0
        k[target, :, 0], v[target] = 3.0 * dim ** 0.5, 9.0

    out, expected = attention_case(pkg, ops, rows=rows, position=position, heads=2, kv_heads=1, dim=dim, vdim=dim, window=window,
                                   kernel=kernel, edit=plant)
    visible = np.array([target <= i < target + window for i in range(position, position + rows)])
    assert_near(out, expected, 0, factor=2.0)
    mean = out.float().cpu().numpy().mean(axis=(1, 2))
    assert (mean[visible] > 6.0).all() and (np.abs(mean[~visible]) < 1.0).all()
    # the query at index 60 is the one whose edge the key lies on
    assert visible[60] == (key_at in ("oldest in the window", "own"))


LATENT = 4


def latent_case(pkg, ops, *, rows, position, heads, rank, window, sinks=True, seed=0, edit=None, kernel=LATENT):
    """Queries against latents that are keys and values; returns (output, expected [rows, heads, rank])."""
    rng = np.random.default_rng(seed)
    total, capacity = position + rows, position + rows + 70
    q, c = rng.normal(0, 1, (rows, heads, rank)), rng.normal(0, 1, (capacity, rank))
    if edit is not None:
        edit(q, c)
    c[total:] = np.nan                                              # what lies behind the last token is never read
    (dq, q), (dc, c) = activation(q, 0), activation(c, 0)
    sink = rng.uniform(-2.0, 4.0, heads).astype(np.float32)
    ds, out = cuda(sink), empty((rows, heads, rank), 0)
    call(ops, "window_attention", pkg.WindowAttention(
        query=dq.data_ptr(), key_cache=dc.data_ptr(), value_cache=dc.data_ptr(), output=out.data_ptr(), rows=rows, position=position,
        capacity=capacity, heads=heads, kv_heads=1, dim=rank, value_dim=rank, window=window, scale=rank ** -0.5, sink=int(sinks),
        sink_logit=ds.data_ptr(), kernel=kernel))
    shared = c[:total, None]
    return out, last_rows(q, shared, shared, scale=rank ** -0.5, window=window, sink=sink if sinks else None)


@pytest.mark.parametrize("kernel", [LATENT, 0])
@pytest.mark.parametrize("sinks", [True, False])
@pytest.mark.parametrize("rank", [64, 128, 192, 256, 320, 384, 448, 512])
def test_latent_kernel(pkg, ops, rank, sinks, kernel):
    for rows, position, heads, window in ((1, 0, 1, 9), (1, 6, 16, 100), (2, 500, 17, 500), (8, 700, 5, 127), (1, 1300, 33, 1024),
                                          (3, 65, 12, 64)):
        out, expected = latent_case(pkg, ops, rows=rows, position=position, heads=heads, rank=rank, window=window, sinks=sinks,
                                    seed=rank + rows, kernel=kernel)
        assert_near(out, expected, 0, factor=2.0)


@pytest.mark.parametrize("target", [0, 1, 62, 63, 64, 65, 127, 300, 511, 512])
def test_one_latent_stands_out(pkg, ops, target):
    """One token far above the rest, at the borders of tiles and of the shares of a cluster, just inside and just
    outside the window."""
    position, window = 600, 537                                      # sees 64 .. 600; the row before it 63 .. 599

    def plant(q, c):
        q *= 0.02
        q[..., 0], c[:, 0] = 4.0, 0.0
        c[target, 0], c[target, 1:] = 40.0, 9.0

    out, expected = latent_case(pkg, ops, rows=2, position=position - 1, heads=3, rank=128, window=window, edit=plant, sinks=False)
    assert_near(out, expected, 0, factor=2.0)
    mean = out.float().cpu().numpy()[..., 1:].mean(axis=(1, 2))
    assert list(mean > 6.0) == [target >= 63, target >= 64]


@TYPES
@pytest.mark.parametrize("rows, heads, dim, vdim, rank", [(1, 3, 24, 40, 72), (2, 5, 128, 128, 512), (4, 1, 1, 3, 1), (7, 4, 33, 7, 51),
                                                         (8, 2, 200, 96, 1000)])
def test_absorbed_heads_equal_expanded_heads(pkg, ops, float32, rows, heads, dim, vdim, rank):
    """Queries against latents and values behind the attention, piece by piece and as a whole, against expanded
    keys and values."""
    rng = np.random.default_rng(rank)
    position, window = 20, 13
    total = position + rows
    q, qv = activation(rng.normal(0, 1, (rows, heads, dim)), float32)
    uk, ukv = activation(rng.normal(0, rank ** -0.5, (heads * dim, rank)), 0)
    uv, uvv = activation(rng.normal(0, rank ** -0.5, (heads * vdim, rank)), 0)
    c, cv = activation(rng.normal(0, 1, (total, rank)), float32)
    absorbed, mixed, out = empty((rows, heads, rank), float32), empty((rows, heads, rank), float32), empty((rows, heads, vdim), float32)
    ops.call("absorb_queries", q.data_ptr(), uk.data_ptr(), rows, heads, dim, rank, absorbed.data_ptr(), float32, stream())
    assert_near(absorbed, np.einsum("rhd,hdc->rhc", qv, ukv.reshape(heads, dim, rank)), float32)
    call(ops, "window_attention", pkg.WindowAttention(
        query=absorbed.data_ptr(), key_cache=c.data_ptr(), value_cache=c.data_ptr(), output=mixed.data_ptr(), rows=rows,
        position=position, capacity=total, heads=heads, kv_heads=1, dim=rank, value_dim=rank, window=window, scale=dim ** -0.5,
        float32=float32))
    ops.call("expand_values", mixed.data_ptr(), uv.data_ptr(), rows, heads, vdim, rank, out.data_ptr(), float32, stream())
    mv = mixed.double().cpu().numpy()
    assert_near(out, np.einsum("rhc,hvc->rhv", mv, uvv.reshape(heads, vdim, rank)), float32)
    keys, values = (cv @ ukv.T).reshape(total, heads, dim), (cv @ uvv.T).reshape(total, heads, vdim)
    expected = oracle.attention(np.concatenate([np.zeros((position, heads, dim)), qv]), keys, values, scale=dim ** -0.5, size=window)
    assert_near(out, expected[position:], float32, factor=2.0)


def test_latent_refusals(pkg, ops):
    x = empty((64, 64), 0)
    with pytest.raises(pkg.OpsError) as error:
        latent_case(pkg, ops, rows=1, position=3, heads=2, rank=72, window=5)
    assert error.value.code == 5
    for rows, rank in ((9, 8), (1, 1025)):
        with pytest.raises(pkg.OpsError) as error:
            ops.call("absorb_queries", x.data_ptr(), x.data_ptr(), rows, 1, 8, rank, x.data_ptr(), 0, stream())
        assert error.value.code == 2
    with pytest.raises(pkg.OpsError) as error:                        # more experts than the kernels hold
        call(ops, "route_rows", pkg.Route(logits=x.data_ptr(), logit_stride=2000, rows=1, experts=1500, top=1, expert=x.data_ptr(),
                                          score=x.data_ptr()))
    assert error.value.code == 2

"""Operators of the decoder graph, each alone, against float64 statements (gigusun_oracle.py): odd and unequal
sizes, both activation types, every kernel behind an operator, keys at every kind of edge."""
from __future__ import annotations

import numpy as np
import pytest

import gigusun_oracle as oracle
from gpu_util import stream

pytestmark = pytest.mark.gpu


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


def assert_near(actual, expected, float32, factor=1.0):
    actual = actual.double().cpu().numpy() if hasattr(actual, "cpu") else actual
    bound = (2e-5 if float32 else 1.2e-2) * factor
    scale = np.sqrt(np.mean(expected * expected)) + 1e-30
    worst = np.max(np.abs(actual - expected) / (np.abs(expected) + scale))
    assert np.isfinite(actual).all() and worst < bound, (worst, bound)


TYPES = pytest.mark.parametrize("float32", [0, 1], ids=["bf16", "f32"])


@TYPES
@pytest.mark.parametrize("width", [8, 60, 77, 1536, 8200, 16392])
def test_row_norms(ops, float32, width):
    rng = np.random.default_rng(width)
    rows, eps = 5, 1e-3
    x = rng.normal(0, 0.05, (rows, width)).astype(np.float32)      # small enough that epsilon matters
    gain = rng.uniform(0.5, 1.5, width).astype(np.float32)
    out = empty((rows, width), float32)
    dx, dg = cuda(x), cuda(gain)
    ops.call("rms_norm_residual", dx.data_ptr(), dg.data_ptr(), rows, width, eps, float32, out.data_ptr(), stream())
    assert_near(out, oracle.rms(x.astype(np.float64), eps) * gain, float32)
    coefficients = np.array([0.7, -0.4, 0.3, 0.2], np.float32)
    z, zv = activation(rng.normal(0, 0.8, (rows, width)), float32)
    dc = cuda(coefficients)
    ops.call("poly_norm", z.data_ptr(), dc.data_ptr(), rows, width, eps, float32, out.data_ptr(), stream())
    assert_near(out, oracle.poly_norm(zv, coefficients.astype(np.float64), eps), float32)
    ops.call("poly_norm", z.data_ptr(), dc.data_ptr(), rows, width, eps, float32, z.data_ptr(), stream())
    assert bool((z == out).all())                                  # in place


@pytest.mark.parametrize("width", [48, 51, 9000])
def test_embedding_adds_the_position_before_its_norm(ops, width):
    import torch

    rng = np.random.default_rng(width)
    table, tv = activation(rng.normal(0, 1, (30, width)), 0)
    places, pv = activation(rng.normal(0, 1, (40, width)), 0)
    gain = rng.uniform(0.5, 1.5, width).astype(np.float32)
    tokens = np.array([3, 29, 0, 3], np.int32)
    out, dt, dg = empty((4, width), 1), cuda(tokens), cuda(gain)
    ops.call("embed_positions", dt.data_ptr(), table.data_ptr(), places.data_ptr(), dg.data_ptr(), 4, width, 30, 36, 1e-6,
             out.data_ptr(), stream())
    expected = oracle.embed(tokens, tv, pv, gain.astype(np.float64) - 1.0, 1e-6, first=36)
    assert_near(out, expected, 1)
    bad = cuda(np.array([1, 30, 2, 2], np.int32))                  # an id outside the vocabulary
    ops.call("embed_positions", bad.data_ptr(), table.data_ptr(), places.data_ptr(), dg.data_ptr(), 4, width, 30, 0, 1e-6,
             out.data_ptr(), stream())
    assert ops.status("check_async_errors", stream()) == 2
    assert not out[1].any() and bool(torch.isfinite(out).all())


def test_distance_table(ops):
    r1, r2 = np.array([0.3, 1.7], np.float32), np.array([0.05, 2.5], np.float32)
    d1, d2, table = cuda(r1), cuda(r2), empty((2, 700), 1)
    ops.call("distance_bias_table", d1.data_ptr(), d2.data_ptr(), 2, 700, table.data_ptr(), stream())
    expected = r1[:, None].astype(np.float64) * np.log1p(r2[:, None].astype(np.float64) * np.arange(700))
    assert_near(table, expected, 1)


@pytest.mark.parametrize("rows", [1, 3, 8, 11, 17, 64, 100, 129, 600])
@pytest.mark.parametrize("inner, outer", [(16, 24), (72, 300), (200, 37), (192, 1032), (128, 8)])
def test_f32_results(ops, rows, inner, outer):
    """F32 multiply-adds, and BF16 operands whose F32 accumulator is stored or added without rounding."""
    rng = np.random.default_rng(rows * 1000 + outer)
    x, xv = activation(rng.normal(0, 1, (rows, inner)), 0)
    w, wv = activation(rng.normal(0, 1, (outer, inner)), 0)
    base = rng.normal(0, 1, (rows, outer)).astype(np.float32)
    exact = cuda(rng.normal(0, 1, (rows, inner)).astype(np.float32))
    work = empty((1 << 22,), 1)
    for accumulate in (0, 1):
        out = cuda(base)
        ops.call("f32_linear", exact.data_ptr(), w.data_ptr(), rows, inner, outer, accumulate, out.data_ptr(), stream())
        assert_near(out, exact.double().cpu().numpy() @ wv.T + accumulate * base, 1)
        for workspace in (None, work.data_ptr()):
            out = cuda(base)
            ops.call("bf16_linear_f32_result", x.data_ptr(), w.data_ptr(), rows, inner, outer, accumulate, workspace,
                     work.numel() * 4, out.data_ptr(), stream())
            ops.call("check_async_errors", stream())
            assert_near(out, xv @ wv.T + accumulate * base, 1)


# ---------------------------------------------------------------- attention
def window_case(pkg, ops, *, rows, position, heads, kv_heads, dim, vdim, window, keep_first, kernel, float32=0, softcap=15.0,
                sink=1, gated=True, biased=True, seed=0, edit=None):
    """Runs one call; returns (output, expected [rows, heads, vdim]).  `edit(q, k, v)` may plant values."""
    rng = np.random.default_rng(seed)
    total, capacity = position + rows, position + rows + 5
    q = rng.normal(0, 1, (rows, heads, dim))
    k = rng.normal(0, 1, (capacity, kv_heads, dim))
    v = rng.normal(0, 1, (capacity, kv_heads, vdim))
    if edit is not None:
        edit(q, k, v)
    k[total:], v[total:] = 1e4, 1e4                                 # what lies behind the last key is never read
    (dq, q), (dk, k), (dv, v) = (activation(x, float32) for x in (q, k, v))
    gate, gv = activation(rng.normal(0, 1, (rows, heads + 3)), float32)
    r1, r2 = rng.uniform(0.1, 0.8, heads), rng.uniform(0.05, 1.0, heads)
    bias = (r1[:, None] * np.log1p(r2[:, None] * np.arange(total))).astype(np.float32)
    db, out = cuda(bias), empty((rows, heads, vdim), float32)
    scale = dim ** -0.5
    import ctypes

    args = pkg.WindowAttention(query=dq.data_ptr(), key_cache=dk.data_ptr(), value_cache=dv.data_ptr(),
                               gate=gate.data_ptr() if gated else None, gate_stride=heads + 3,
                               distance_bias=db.data_ptr() if biased else None, bias_stride=total, output=out.data_ptr(),
                               rows=rows, position=position, capacity=capacity, heads=heads, kv_heads=kv_heads, dim=dim,
                               value_dim=vdim, window=window, keep_first=keep_first, scale=scale, softcap=softcap, sink=sink,
                               float32=float32, kernel=kernel)
    ops.call("window_attention", ctypes.addressof(args), stream())
    ops.call("check_async_errors", stream())
    expected = np.zeros((rows, heads, vdim))
    for r in range(rows):
        i = position + r
        seen = oracle.visible_keys(i, window if window else i + 1, keep_first)
        for h in range(heads):
            s = (k[seen, h // (heads // kv_heads)] @ q[r, h]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            if biased:
                s = s - r1[h] * np.log1p(r2[h] * (i - seen))
            p = oracle.softmax_with_sink(s) if sink else np.exp(s - s.max()) / np.exp(s - s.max()).sum()
            expected[r, h] = p @ v[seen, h // (heads // kv_heads)]
        if gated:
            expected[r] *= oracle.sigmoid(gv[r, :heads])[:, None]
    return out, expected


ROW, TILE, TENSOR = 1, 2, 3


@TYPES
@pytest.mark.parametrize("kernel", [ROW, TILE], ids=["row", "tile"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim", [(6, 2, 40, 24), (3, 1, 17, 5), (4, 4, 200, 136), (2, 1, 96, 256),
                                                         (8, 2, 64, 72)])
def test_attention_sizes(pkg, ops, float32, kernel, heads, kv_heads, dim, vdim):
    for rows, position in ((1, 0), (1, 61), (7, 30), (45, 3)):
        out, expected = window_case(pkg, ops, rows=rows, position=position, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                                    window=21, keep_first=3, kernel=kernel, float32=float32, seed=rows)
        assert_near(out, expected, float32)


@pytest.mark.parametrize("dim, vdim", [(64, 64), (96, 96), (128, 72), (72, 128), (128, 128)])
@pytest.mark.parametrize("rows, position, window, keep_first", [
    (1, 0, 7, 0), (130, 0, 64, 4), (200, 0, 0, 0), (150, 300, 96, 6), (64, 500, 65, 70), (300, 1, 128, 1), (129, 63, 1, 0),
    (257, 700, 200, 129)])
def test_attention_tensor_cores(pkg, ops, dim, vdim, rows, position, window, keep_first):
    out, expected = window_case(pkg, ops, rows=rows, position=position, heads=4, kv_heads=2, dim=dim, vdim=vdim, window=window,
                                keep_first=keep_first, kernel=TENSOR)
    assert_near(out, expected, 0, factor=2.0)                       # the probabilities are BF16 operands as well


@pytest.mark.parametrize("kernel", [ROW, TILE, TENSOR])
@pytest.mark.parametrize("softcap, sink, gated, biased", [(0.0, 1, True, True), (90.0, 1, True, True), (1.5, 1, True, True), (3.0, 0, True, True), (15.0, 1, False, True),
                                                           (15.0, 1, True, False), (0.0, 0, False, False)])
def test_attention_options(pkg, ops, kernel, softcap, sink, gated, biased):
    out, expected = window_case(pkg, ops, rows=70, position=90, heads=4, kv_heads=1, dim=64, vdim=80, window=33, keep_first=2,
                                kernel=kernel, softcap=softcap, sink=sink, gated=gated, biased=biased)
    assert_near(out, expected, 0)


@pytest.mark.parametrize("kernel", [ROW, TILE, TENSOR])
@pytest.mark.parametrize("key_at", ["oldest in the window", "just outside", "last kept", "first after the kept", "own", "next"])
def test_one_key_stands_out(pkg, ops, kernel, key_at):
    """One key that every query scores far above the rest, at the edges of what a query sees: its value dominates
    exactly where it is visible."""
    rows, position, window, keep = 140, 200, 50, 5
    target = {"oldest in the window": position + 60 - window + 1, "just outside": position + 60 - window,
              "last kept": keep - 1, "first after the kept": keep, "own": position + 60, "next": position + 61}[key_at]

    def plant(q, k, v):
        q[..., 0], k[..., 0] = 4.0, 0.0
        k[target, :, 0], v[target] = 20.0, 9.0

    out, expected = window_case(pkg, ops, rows=rows, position=position, heads=4, kv_heads=2, dim=64, vdim=64, window=window,
                                keep_first=keep, kernel=kernel, gated=False, softcap=30.0, edit=plant)
    visible = np.array([target <= i and (i - target < window or target < keep) for i in range(position, position + rows)])
    assert_near(out, expected, 0)
    mean = out.float().cpu().numpy().mean(axis=(1, 2))
    assert (mean[visible] > 3.0).all() and (np.abs(mean[~visible]) < 1.0).all()
    # the query at index 60 is the one whose edge the key lies on
    assert visible[60] == (key_at in ("oldest in the window", "last kept", "own"))


@pytest.mark.parametrize("kernel", [ROW, TILE, TENSOR])
def test_the_sink_alone(pkg, ops, kernel):
    """Scores far below zero leave almost everything to the sink."""
    def plant(q, k, v):
        q[..., 0], k[..., 0], v[:] = 10.0, -20.0, 5.0

    out, expected = window_case(pkg, ops, rows=66, position=10, heads=2, kv_heads=1, dim=64, vdim=64, window=16, keep_first=1,
                                kernel=kernel, gated=False, softcap=12.0, edit=plant)
    assert np.abs(out.float().cpu().numpy()).max() < 1e-2 and np.abs(expected).max() < 1e-2


def test_attention_refusals(pkg, ops):
    with pytest.raises(pkg.OpsError) as error:
        window_case(pkg, ops, rows=40, position=0, heads=2, kv_heads=1, dim=40, vdim=64, window=8, keep_first=0, kernel=TENSOR)
    assert error.value.code == 5
    for size in ("dim", "vdim"):                                     # wide heads run in the row kernel only
        with pytest.raises(pkg.OpsError) as error:
            window_case(pkg, ops, **(dict(rows=2, position=0, heads=2, kv_heads=1, dim=16, vdim=16, window=8, keep_first=0,
                                          kernel=TILE) | {size: 300}))
        assert error.value.code == 5
    for bad in (dict(heads=3, kv_heads=2), dict(dim=1032), dict(softcap=-1.0)):
        case = dict(rows=2, position=0, heads=2, kv_heads=1, dim=16, vdim=16, window=8, keep_first=0, kernel=0) | bad
        with pytest.raises(pkg.OpsError) as error:
            window_case(pkg, ops, **case)
        assert error.value.code == 2


@TYPES
@pytest.mark.parametrize("dim, vdim", [(40, 24), (17, 33), (128, 200)])
def test_head_norms_and_cache_rows(pkg, ops, float32, dim, vdim):
    import ctypes

    rng = np.random.default_rng(dim)
    rows, position, capacity, heads, kv_heads, eps = 5, 7, 14, 6, 2, 1e-2
    key_column = heads * dim + 3
    value_column = key_column + kv_heads * dim + 1
    stride = value_column + kv_heads * vdim + 9
    x, xv = activation(rng.normal(0, 0.3, (rows, stride)), float32)
    gq, gk = (rng.uniform(0.5, 1.5, dim).astype(np.float32) for _ in range(2))
    dq, dk = cuda(gq), cuda(gk)
    query, keys, values = (empty(s, float32) for s in ((rows, heads, dim), (capacity, kv_heads, dim), (capacity, kv_heads, vdim)))
    args = pkg.HeadNorm(projection=x.data_ptr(), stride=stride, key_column=key_column, value_column=value_column,
                        query_gain=dq.data_ptr(), key_gain=dk.data_ptr(), query=query.data_ptr(), key_cache=keys.data_ptr(),
                        value_cache=values.data_ptr(), rows=rows, position=position, capacity=capacity, heads=heads,
                        kv_heads=kv_heads, dim=dim, value_dim=vdim, epsilon=eps, float32=float32)
    ops.call("head_norm_append", ctypes.addressof(args), stream())
    assert_near(query, oracle.rms(xv[:, :heads * dim].reshape(rows, heads, dim), eps) * gq, float32)
    assert_near(keys[position:position + rows],
                oracle.rms(xv[:, key_column:key_column + kv_heads * dim].reshape(rows, kv_heads, dim), eps) * gk, float32)
    assert bool((values[position:position + rows].reshape(rows, -1) ==
                 x[:, value_column:value_column + kv_heads * vdim]).all())
    assert bool(keys[:position].isnan().all()) and bool(values[position + rows:].isnan().all())   # neighbours untouched
    args.position = capacity - rows + 1
    assert ops.status("head_norm_append", ctypes.addressof(args), stream()) == 2


# ---------------------------------------------------------------- recurrences
class Recurrence:
    """One recurrent mixer with random inputs; run() pushes the next rows through it."""

    def __init__(self, pkg, ops, *, delta, rows, heads, kv_heads, dim, vdim, float32, taps=4, rank=5, tau=9.0, seed=0,
                 projection_scale=1.0):
        self.pkg, self.ops = pkg, ops
        rng = np.random.default_rng(seed)
        up = lambda n: (n + 7) // 8 * 8
        self.delta, self.heads, self.kv_heads, self.dim, self.vdim, self.float32 = delta, heads, kv_heads, dim, vdim, float32
        qk = (kv_heads if delta else heads) * dim
        self.key_column = up(qk)
        self.value_column = self.key_column + up(qk)
        self.gate_column = self.value_column + up(heads * vdim)
        self.beta_column = self.gate_column + up(heads * vdim)
        self.decay_column = self.beta_column + up(heads if delta else rank)
        self.stride = self.decay_column + (up(heads) if delta else 0)
        self.taps, self.rank, self.tau, self.eps = taps, rank, tau, 1e-5
        self.projection, self.values = activation(rng.normal(0, projection_scale, (rows, self.stride)), float32)
        f32 = lambda *shape, low=-1.0, high=1.0: rng.uniform(low, high, shape).astype(np.float32)
        self.conv, self.rate, self.shift = f32(self.gate_column, taps), -np.exp(f32(heads, low=-3.0)), f32(heads)
        self.weight, self.bias, self.norm = f32(rank, heads * dim), f32(heads * dim, high=4.0), f32(vdim, low=0.5, high=1.5)
        self.device = [cuda(x) for x in (self.conv, self.rate, self.shift, self.weight, self.bias, self.norm)]
        self.state = empty((heads, dim, vdim), 1)
        self.history = empty((max(1, taps - 1), self.gate_column), float32)
        self.at = 0

    def run(self, rows):
        import ctypes

        conv, rate, shift, weight, bias, norm = self.device
        size = self.ops.lib.evo_b200_recurrent_workspace_bytes(int(self.delta), rows, self.heads, self.kv_heads, self.dim,
                                                               self.vdim, self.float32)
        work, out = empty((size // 4 + 1,), 1), empty((rows, self.heads * self.vdim), self.float32)
        part = self.projection[self.at:self.at + rows].contiguous()
        args = self.pkg.Recurrent(
            delta=int(self.delta), projection=part.data_ptr(), stride=self.stride, key_column=self.key_column,
            value_column=self.value_column, gate_column=self.gate_column, beta_column=self.beta_column,
            decay_column=self.decay_column, rows=rows, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim,
            value_dim=self.vdim, conv=conv.data_ptr(), conv_taps=self.taps, conv_history=self.history.data_ptr(),
            decay_rate=rate.data_ptr(), decay_shift=shift.data_ptr(), decay_weight=weight.data_ptr(),
            decay_bias=bias.data_ptr(), decay_rank=self.rank, tau=self.tau, output_norm=norm.data_ptr(), epsilon=self.eps,
            state=self.state.data_ptr(), fresh=int(self.at == 0), workspace=work.data_ptr(), output=out.data_ptr(),
            float32=self.float32)
        self.ops.call("recurrent_mixer", ctypes.addressof(args), stream())
        self.ops.call("check_async_errors", stream())
        self.at += rows
        return out

    def restart(self):
        self.at = 0

    def expected(self, rows):
        x, H, G, dim, vdim = self.values[:rows], self.heads, self.kv_heads, self.dim, self.vdim
        cut = lambda column, n, shape: x[:, column:column + n].reshape(rows, *shape)
        gate = cut(self.gate_column, H * vdim, (H, vdim))
        if self.delta:
            mixed = oracle.silu(oracle.causal_convolution(x[:, :self.gate_column], self.conv.astype(np.float64)))
            q = oracle.unit_vectors(mixed[:, :G * dim].reshape(rows, G, dim)) * dim ** -0.5
            k = oracle.unit_vectors(mixed[:, self.key_column:self.key_column + G * dim].reshape(rows, G, dim))
            v = mixed[:, self.value_column:self.value_column + H * vdim].reshape(rows, H, vdim)
            beta = oracle.sigmoid(cut(self.beta_column, H, (H,)))
            g = np.exp(self.rate.astype(np.float64) * oracle.softplus(cut(self.decay_column, H, (H,)) + self.shift))
            o, state = oracle.gated_delta_rule(q, k, v, beta, g)
        else:
            q = cut(0, H * dim, (H, dim)) * dim ** -0.5
            k, v = cut(self.key_column, H * dim, (H, dim)), cut(self.value_column, H * vdim, (H, vdim))
            z = cut(self.beta_column, self.rank, (self.rank,)) @ self.weight.astype(np.float64) + self.bias
            alpha = np.exp(-oracle.softplus(-z) / self.tau).reshape(rows, H, dim)
            o, state = oracle.gated_linear_attention(q, k, v, alpha)
        return (oracle.rms(o, self.eps) * self.norm * oracle.silu(gate)).reshape(rows, -1), state


RECURRENT_SIZES = [(4, 2, 28, 20), (3, 3, 5, 33), (6, 1, 64, 40), (2, 2, 96, 17), (4, 1, 128, 64), (2, 1, 200, 24)]


@TYPES
@pytest.mark.parametrize("delta", [False, True], ids=["linear", "delta"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim", RECURRENT_SIZES)
def test_recurrences(pkg, ops, float32, delta, heads, kv_heads, dim, vdim):
    rows = 150
    case = Recurrence(pkg, ops, delta=delta, rows=rows, heads=heads, kv_heads=kv_heads if delta else heads, dim=dim, vdim=vdim,
                      float32=float32, taps=1 + dim % 5)
    expected, state = case.expected(rows)
    assert_near(case.run(rows), expected, float32, factor=4.0)
    assert_near(case.state, state, float32 or not delta)            # (BF16 rounds the convolved values, not the state)


@pytest.mark.parametrize("delta", [False, True], ids=["linear", "delta"])
@pytest.mark.parametrize("taps", [1, 2, 6])
@pytest.mark.parametrize("portions", [[2] * 30, [1] * 60, [16, 1, 17, 2, 24], [3, 57], [60], [5, 4, 1, 1, 1, 48]])
def test_recurrences_in_portions(pkg, ops, delta, taps, portions):
    """The state and the convolution's history carry over any cut; a restart forgets both."""
    case = Recurrence(pkg, ops, delta=delta, rows=60, heads=4, kv_heads=2 if delta else 4, dim=36, vdim=40, float32=1, taps=taps,
                      seed=3)
    expected, state = case.expected(60)
    for _ in range(2):
        parts = [case.run(n).cpu().numpy() for n in portions]
        assert_near(np.concatenate(parts).astype(np.float64), expected, 1, factor=4.0)
        assert_near(case.state, state, 1)
        case.restart()


@pytest.mark.parametrize("delta", [False, True], ids=["linear", "delta"])
def test_a_lost_state_would_show(pkg, ops, delta):
    """Slow decays: what the first tokens wrote still dominates far away."""
    case = Recurrence(pkg, ops, delta=delta, rows=300, heads=2, kv_heads=2, dim=32, vdim=16, float32=1, seed=5, tau=4000.0,
                      projection_scale=0.3)
    case.rate[:] = -1e-4
    case.device[1].copy_(cuda(case.rate))
    expected, _ = case.expected(300)
    out = np.concatenate([case.run(n).cpu().numpy() for n in (100, 1, 150, 49)]).astype(np.float64)
    assert_near(out, expected, 1, factor=6.0)
    case.restart()
    case.run(100)
    case.at = 0                                                     # forget the state: a fresh start at row 100
    case.projection = case.projection[100:].contiguous()
    forgotten = case.run(200).double().cpu().numpy()
    assert np.abs(forgotten[-50:] - expected[-50:]).max() > 1e-2


def test_extreme_gates_stay_finite(pkg, ops):
    for delta in (False, True):
        case = Recurrence(pkg, ops, delta=delta, rows=40, heads=2, kv_heads=2, dim=24, vdim=16, float32=1, projection_scale=60.0,
                          tau=0.5)
        expected, _ = case.expected(40)
        out = case.run(40).double().cpu().numpy()
        assert np.isfinite(out).all() and np.isfinite(expected).all()
        assert_near(out, expected, 1, factor=50.0)

"""The kernels of the Dalorax models, and the engine on them, against the plain restatement (``oracle_mixers``): each
mechanism alone, then whole models in prompts, portions, decoding, batches and generation."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

import oracle_mixers as plain
from mixer_models import (SANDWICHES, bf16_round, dense_mlp, routed_mlp, sandwich_config, settled_tokens, weights_of,
                          window_layer)
from test_gpu_mixers import DTYPES, Reference as AnyReference, build, close, download, empty, greedy, logit_error, suffix, upload
from test_mixers_cpu import write_checkpoint

pytestmark = pytest.mark.gpu


class Reference(AnyReference):
    """Bounded norms on every path keep the rounding errors of these models even: one limit for all places."""

    LIMIT = {"float32": 2e-6, "bfloat16": 6e-3}

    def limit(self, dtype):
        return np.full(len(self.tokens), self.LIMIT[dtype])


def run(runtime, name, buffers, parameters):
    runtime.dispatch(name, buffers=buffers, parameters=parameters)


# ---- products ------------------------------------------------------------------------------------------

SHAPES = [(1, 24, 104), (2, 6, 50), (3, 78, 50), (8, 130, 200), (9, 64, 72), (17, 40, 1000), (33, 96, 128), (64, 334, 264),
          (65, 80, 104), (130, 200, 256), (257, 520, 336), (300, 62, 50), (200, 1026, 64), (1, 16, 4096), (140, 32, 1024)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k", SHAPES)
def test_paired_columns_and_scale(runtime, dtype, m, n, k):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(m * 1000 + n)
    x, w = bf16_round(rng.standard_normal((m, k))), bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    bias = rng.standard_normal(n).astype(np.float32)
    y = x.astype(np.float64) @ w.T.astype(np.float64)
    absent = empty(runtime, 4)
    for has_bias, scale in ((False, 1.0), (True, 0.3)):
        z = y * scale + (bias if has_bias else 0.0)
        out = empty(runtime, m * n // 2, dtype)
        run(runtime, "llmopt_dense_linear_" + suffix(dtype),
            [upload(runtime, x, dtype), upload(runtime, w, dtype), upload(runtime, bias), out, absent, absent, absent],
            parameters.dense_linear(m=m, n=n, k=k, split=n, has_bias=has_bias, epilogue="silu_pair", scale=scale))
        close(download(out, (m, n // 2), dtype), plain.silu(z[:, ::2]) * z[:, 1::2], 6e-3 if dtype == "bfloat16" else 3e-6)
    out32 = empty(runtime, m * n)
    run(runtime, "llmopt_dense_linear_" + suffix(dtype),
        [upload(runtime, x, dtype), upload(runtime, w, dtype), absent, absent, out32, absent, absent],
        parameters.dense_linear(m=m, n=n, k=k, split=0, scale=-2.5))
    close(download(out32, (m, n)), -2.5 * y, 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sequences,tokens,k,own,heads,dim,vdim,extra", [
    (1, 1, 104, 48, 3, 24, 40, 0), (5, 1, 64, 30, 2, 18, 10, 3), (1, 2, 50, 7, 1, 9, 13, 1), (1, 64, 128, 96, 2, 64, 64, 0),
    (1, 65, 128, 96, 2, 64, 64, 0), (1, 150, 96, 130, 3, 40, 24, 5), (2, 100, 72, 64, 1, 32, 136, 40), (1, 300, 256, 0, 8, 8, 8, 0)])
def test_keys_and_values_straight_into_the_cache(runtime, dtype, sequences, tokens, k, own, heads, dim, vdim, extra):
    from llmopt_b200 import parameters
    from llmopt_b200.kv_cache import RowLayout

    rng = np.random.default_rng(tokens)
    m, keys, values = sequences * tokens, heads * dim, heads * vdim
    n = own + keys + values + extra
    x, w = bf16_round(rng.standard_normal((m, k))), bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    bias = rng.standard_normal(n).astype(np.float32)
    layout = RowLayout([(1, 8, 16), (heads, dim, vdim), (1, 3, 3)])
    region, stride, slots, rows = layout.regions[1], 400, 900, sequences + 2
    order = rng.permutation(slots)[:rows * stride // 3]
    table = np.zeros((rows, stride), np.uint32)
    for row in range(rows):
        table[row, :len(order) // rows] = order[row * (len(order) // rows):][:len(order) // rows]
    if tokens > len(order) // rows - 30:
        table[2, :] = rng.permutation(slots)[:stride]
    which = (rng.permutation(rows)[:sequences] if tokens == 1 or sequences > 1 else np.array([2])).astype(np.uint32)
    past = rng.integers(0, 30, size=sequences).astype(np.uint32)
    before = bf16_round(rng.standard_normal((slots, layout.token_elements)))
    pool = upload(runtime, before, dtype)
    out, out32 = empty(runtime, max(m * own, 1), dtype), empty(runtime, max(m * extra, 1))
    run(runtime, "llmopt_dense_cached_" + suffix(dtype),
        [upload(runtime, x, dtype), upload(runtime, w, dtype), upload(runtime, bias), out, out32, pool, upload(runtime, table),
         upload(runtime, past), upload(runtime, which)],
        parameters.dense_cached(m=m, n=n, k=k, split=own, tokens=tokens, key_columns=keys, value_columns=values, has_bias=True,
                                token_stride=layout.token_elements, key_offset=region.key_offset, value_offset=region.value_offset,
                                table_stride=stride, table_rows=rows, pool_rows=slots))
    y = x.astype(np.float64) @ w.T.astype(np.float64) + bias
    tolerance = 6e-3 if dtype == "bfloat16" else 3e-6
    if own:
        close(download(out, (m, own), dtype), y[:, :own], tolerance, "rows")
    if extra:
        close(download(out32, (m, extra)), y[:, n - extra:], 1e-5, "fp32 rows")
    want = before.astype(np.float64)
    for row in range(m):
        slot = table[which[row // tokens], past[row // tokens] + row % tokens]
        want[slot, region.key_offset:region.key_offset + keys] = y[row, own:own + keys]
        want[slot, region.value_offset:region.value_offset + values] = y[row, own + keys:own + keys + values]
    got = download(pool, (slots, layout.token_elements), dtype)
    close(got, want, tolerance, "cache")
    untouched = np.ones(before.shape, bool)
    for row in range(m):
        untouched[table[which[row // tokens], past[row // tokens] + row % tokens]] = False
    assert np.array_equal(got[untouched], before[untouched])


def norm_vector(rng, width):
    w, b, alpha = rng.uniform(0.5, 2.0, size=width), rng.standard_normal(width), rng.uniform(0.2, 1.5)
    vector = np.concatenate([w, b, [alpha]]).astype(np.float32)
    named = {"n": vector[:width], "n.b": vector[width:2 * width], "n.alpha": vector[2 * width:]}
    return vector, lambda x: plain.tanh_norm(x, named, "n")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k", SHAPES + [(70, 51, 64), (5, 51, 64), (1, 4096, 256)])
def test_product_that_ends_a_sublayer(runtime, dtype, m, n, k):
    """Norm of the sum, residual in place, the next norm; sums from tiny to far into saturation."""
    from llmopt_b200 import parameters

    rng = np.random.default_rng(m + n)
    x, w = bf16_round(rng.standard_normal((m, k))), bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    x *= 10.0 ** rng.integers(-3, 2, size=(m, 1))
    x = bf16_round(x)
    residual, bias = rng.standard_normal((m, n)) * 3, rng.standard_normal(n).astype(np.float32)
    (post, post_norm), (after, next_norm) = norm_vector(rng, n), norm_vector(rng, n)
    y = x.astype(np.float64) @ w.T.astype(np.float64)
    for has_bias in (False, True):
        kept, out = upload(runtime, residual), empty(runtime, m * n, dtype)
        run(runtime, "llmopt_dense_residual_" + suffix(dtype),
            [upload(runtime, x, dtype), upload(runtime, w, dtype), upload(runtime, bias), upload(runtime, post), upload(runtime, after),
             kept, out], parameters.dense_residual(m=m, n=n, k=k, has_bias=has_bias))
        want = residual.astype(np.float32) + post_norm(y + (bias if has_bias else 0.0))
        close(download(kept, (m, n)), want, 3e-6, "residual")
        close(download(out, (m, n), dtype), next_norm(want), 5e-3 if dtype == "bfloat16" else 3e-6, "next input")


def test_tanh_near_zero_keeps_its_digits(runtime):
    """With a large weight a tiny argument's relative error would show."""
    from llmopt_b200 import parameters

    values = np.concatenate([[0.0], np.geomspace(1e-6, 1e6, 255)]).astype(np.float32)
    values[1::2] *= -1
    identity = np.eye(8, dtype=np.float32)
    x = np.zeros((256, 8), np.float32)
    x[:, 3] = values
    norm = np.zeros(17, np.float32)
    norm[:8], norm[16] = 1.0, 1.0
    kept, out = upload(runtime, np.zeros((256, 8))), empty(runtime, 256 * 8)
    run(runtime, "llmopt_dense_residual_f32",
        [upload(runtime, x), upload(runtime, identity), upload(runtime, norm), upload(runtime, norm), upload(runtime, norm), kept, out],
        parameters.dense_residual(m=256, n=8, k=8))
    got, want = download(kept, (256, 8))[:, 3].astype(np.float64), np.tanh(values.astype(np.float64))
    assert np.max(np.abs(got - want)) < 2e-7
    assert np.max(np.abs(got - want)[1:] / np.abs(want[1:])) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [104, 51, 1, 2, 1028, 700])
def test_embedding_with_sinusoidal_positions(runtime, dtype, width):
    """Also where positions are so late that a 32-bit angle would be off."""
    from llmopt_b200 import parameters

    rng = np.random.default_rng(width)
    table = bf16_round(rng.standard_normal((30, width)))
    norm, next_norm = norm_vector(rng, width)
    turns = 10000.0 ** (-2.0 * np.arange((width + 1) // 2) / width) / (2.0 * np.pi)
    for sequences, tokens in ((1, 1), (3, 1), (1, 70), (2, 5)):
        past = rng.integers(0, 300000, size=sequences).astype(np.uint32)
        past[0] = 0 if tokens == 70 else 262143
        ids = rng.integers(0, 30, size=sequences * tokens)
        x, normed = empty(runtime, sequences * tokens * width), empty(runtime, sequences * tokens * width, dtype)
        run(runtime, "llmopt_embedding_sinusoid_" + suffix(dtype),
            [upload(runtime, ids.astype(np.int64)), upload(runtime, table, dtype), upload(runtime, past),
             upload_f64(runtime, turns), upload(runtime, norm), x, normed],
            parameters.embedding_sinusoid(rows=sequences * tokens, tokens=tokens, vocabulary=30, width=width))
        places = (past[:, None].astype(np.int64) + np.arange(tokens)[None, :]).reshape(-1)
        want = table[ids] + plain.sinusoids(places, width)
        assert np.max(np.abs(download(x, want.shape) - want)) < 1e-6
        after = next_norm(want)
        assert np.max(np.abs(download(normed, want.shape, dtype) - after)) < (5e-3 if dtype == "bfloat16" else 3e-6) * max(1, np.max(np.abs(after)))


def upload_f64(runtime, array):
    from llmopt_b200.cuda_native import Buffer

    return Buffer.of_array(runtime, np.ascontiguousarray(array, np.float64))


@pytest.mark.parametrize("dtype", DTYPES)
def test_gather_rows(runtime, dtype):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(0)
    for width in (5, 104, 1028):
        x, chosen = bf16_round(rng.standard_normal((9, width))), np.array([8, 0, 3, 3, 1], np.uint32)
        out = empty(runtime, 5 * width, dtype)
        run(runtime, "llmopt_gather_rows_" + suffix(dtype), [upload(runtime, x, dtype), upload(runtime, chosen), out],
            parameters.gather_rows(count=5, source_rows=9, width=width))
        assert np.array_equal(download(out, (5, width), dtype), x[chosen])


# ---- attention -----------------------------------------------------------------------------------------

class WindowBench:
    """The attention kernel alone over scattered slots.  The whole sequence's keys and values lie in the cache from the
    start, so that a look into the future shows."""

    def __init__(self, runtime, dtype, q, k, v, *, scale, window=None, keep_first=0, softcap=None, gates=None, weights32=True, seed=0):
        from llmopt_b200.kv_cache import RowLayout

        rng = np.random.default_rng(seed)
        self.runtime, self.dtype, self.q, self.gates = runtime, dtype, q, gates
        tokens, self.kv_heads, self.dim = k.shape
        self.heads, self.vdim, self.tokens = q.shape[1], v.shape[2], tokens
        layout = RowLayout([(1, 8, 8), (self.kv_heads, self.dim, self.vdim), (2, 16, 8)])
        region, slots = layout.regions[1], tokens + 40
        order = rng.permutation(slots)[:tokens]
        pool = bf16_round(rng.standard_normal((slots, layout.token_elements)) * 50.0)
        pool[order, region.key_offset:region.key_offset + self.kv_heads * self.dim] = k.reshape(tokens, -1)
        pool[order, region.value_offset:region.value_offset + self.kv_heads * self.vdim] = v.reshape(tokens, -1)
        table = np.zeros((3, tokens), np.uint32)
        table[1] = order
        self.pool, self.table = upload(runtime, pool, dtype), upload(runtime, table)
        self.row = upload(runtime, np.array([1], np.uint32))
        self.size = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                         token_stride=layout.token_elements, key_offset=region.key_offset, value_offset=region.value_offset,
                         table_stride=tokens, table_rows=3, pool_rows=slots, scale=scale, softcap=softcap or 0.0,
                         window=window or 0, keep_first=keep_first, sink=False, weights32=weights32)
        places = np.arange(tokens)
        mask = {"size": window, "keep_first": keep_first} if window else None
        self.want = plain.masked_attention(*(a.astype(np.float64) for a in (q, k, v)), plain.visible_keys(places, places, mask), scale,
                                           softcap)
        if gates is not None:
            self.want = self.want * plain.sigmoid(gates.astype(np.float64))

    def run(self, first, end, splits=1):
        from llmopt_b200 import parameters

        count, lead = end - first, 8 if self.dim % 8 == 0 else 3
        queries, values = self.heads * self.dim, self.heads * self.vdim
        gates = self.gates if self.gates is not None else np.zeros((self.tokens, self.heads, self.vdim))
        rows = np.concatenate([np.full((count, lead), 9.0), self.q[first:end].reshape(count, -1), gates[first:end].reshape(count, -1)], axis=1)
        projected, out = upload(self.runtime, rows, self.dtype), empty(self.runtime, count * values, self.dtype)
        scratch = empty(self.runtime, 64 + self.kv_heads * splits * (32 + 16 * 256))
        gate = dict(gate_stride=rows.shape[1], gate_column=lead + queries) if self.gates is not None else {}
        for _ in range(2):
            run(self.runtime, "llmopt_row_attention_" + suffix(self.dtype),
                [projected, self.pool, self.table, upload(self.runtime, np.array([first], np.uint32)), self.row, out, scratch, projected],
                parameters.row_attention(sequences=1, tokens=count, splits=splits, query_stride=rows.shape[1], query_column=lead,
                                         **self.size, **gate))
        return download(out, (count, self.heads, self.vdim), self.dtype)

    def check(self, first, end, splits=1, tolerance=None, label=""):
        tolerance = tolerance or (1.2e-2 if self.dtype == "bfloat16" else 5e-6)
        close(self.run(first, end, splits), self.want[first:end], tolerance, f"{label} rows {first} to {end}, {splits} splits")


ATTENTION = {  # heads, key/value heads, dim, vdim
    "gqa": (6, 3, 24, 40), "square64": (4, 2, 64, 64), "square128": (8, 1, 128, 128), "wide": (2, 2, 72, 200),
    "narrow": (16, 1, 48, 32), "many": (20, 1, 32, 48), "odd": (9, 3, 18, 10)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ATTENTION))
@pytest.mark.parametrize("window,keep_first", [(None, 0), (1, 0), (1, 3), (7, 2), (40, 6), (64, 64), (65, 1), (100, 130), (500, 4)])
def test_windows_in_portions(runtime, dtype, name, window, keep_first):
    heads, kv_heads, dim, vdim = ATTENTION[name]
    rng = np.random.default_rng(dim)
    counts = [1, 2, 70, 3, 64, 1, 1, 90, 2, 5, 1]
    total = sum(counts)
    q, k, v = (bf16_round(rng.standard_normal(s)) for s in ((total, heads, dim), (total, kv_heads, dim), (total, kv_heads, vdim)))
    bench = WindowBench(runtime, dtype, q, k, v, scale=1.5 / np.sqrt(dim), window=window, keep_first=keep_first, softcap=4.0,
                        gates=bf16_round(rng.standard_normal((total, heads, vdim))))
    at = 0
    for index, count in enumerate(counts):
        bench.check(at, at + count, splits=[1, 7, 33][index % 3])
        at += count
    bench.check(0, total, label="whole")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep_first", [(40, 6), (64, 0), (129, 64), (16, 17), (300, 1)])
def test_a_key_just_inside_and_just_outside(runtime, dtype, window, keep_first):
    """One key stands out for every query; it must be found exactly where it is visible."""
    rng = np.random.default_rng(window)
    total, heads, dim, vdim = 420, 4, 64, 64
    for place in sorted({0, keep_first - 1, keep_first, keep_first + 1, 63, 64, 100, 127, 128} & set(range(total))):
        mark = rng.standard_normal(dim)
        mark *= 8.0 / np.linalg.norm(mark)
        q = bf16_round(mark + 0.05 * rng.standard_normal((total, heads, dim)))
        k = 0.2 * rng.standard_normal((total, 1, dim))
        k[place, 0] = mark
        v = 0.1 * rng.standard_normal((total, 1, vdim))
        v[place, 0] += 5.0
        bench = WindowBench(runtime, dtype, q, bf16_round(k), bf16_round(v), scale=0.25, window=window, keep_first=keep_first, softcap=15.0)
        found = bench.want[:, 0].mean(axis=1) > 2.5
        expected = np.array([t >= place and (t - place < window or place < keep_first) for t in range(total)])
        assert np.array_equal(found, expected)
        bench.check(0, total, label=f"key {place}")
        for edge in (place, place + window - 1, place + window, total - 1):
            if place <= edge < total:
                bench.check(edge, edge + 1, splits=1 + edge % 5, label=f"key {place}")
            if 0 < edge < total - 1:
                bench.check(edge - 1, edge + 1, splits=3, label=f"key {place}")
                bench.check(edge - 1, min(edge + 66, total), label=f"key {place}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 20, 90])
def test_score_cap(runtime, dtype, tokens):
    """Scores far beyond the cap: all but equal weights, where the uncapped ones would pick a single key."""
    rng = np.random.default_rng(tokens)
    total = 90
    q, k, v = (bf16_round(rng.standard_normal((total, n, 32)) * s) for n, s in ((2, 4.0), (1, 4.0), (1, 1.0)))
    for cap in (0.5, 6.0, 50.0, None):
        bench = WindowBench(runtime, dtype, q, k, v, scale=1.0, softcap=cap)
        bench.check(total - tokens, total, splits=3 if tokens == 1 else 1, tolerance=None if dtype == "bfloat16" else 2e-5)


def test_softmax_weights_meet_the_values_in_32_bits(runtime):
    """Large values of alternating sign: the sums are small, and rounded weights would leave their rounding behind."""
    rng = np.random.default_rng(2)
    total = 128
    q, k = bf16_round(0.3 * rng.standard_normal((total, 4, 64))), bf16_round(rng.standard_normal((total, 1, 64)))
    k[1::2] = k[::2]
    v = np.empty((total, 1, 64), np.float32)
    v[::2] = bf16_round(64.0 + 32.0 * rng.random((total // 2, 1, 64)))
    v[1::2] = -v[::2]
    v += bf16_round(0.5 * rng.integers(0, 2, size=v.shape))
    v = bf16_round(v)
    for first, end in ((total - 2, total), (total - 1, total), (64, total)):
        rough, fine = (np.max(np.abs(WindowBench(runtime, "bfloat16", q, k, v, scale=0.2, weights32=flag).run(first, end) -
                                     (want := WindowBench(runtime, "bfloat16", q, k, v, scale=0.2).want[first:end]))[:, :, 0])
                       for flag in (False, True))
        scale = np.max(np.abs(want))
        assert fine <= 6e-3 * scale and np.isfinite(rough), (fine / scale, rough / scale)


def test_queries_alone_are_prepared(runtime):
    """A layer without keys of its own: head norm and rotation of the queries, and the cache stays as it is."""
    from llmopt_b200 import parameters
    from llmopt_b200.model import RotarySpec
    from llmopt_b200.quantize import rotary_pairs

    rng = np.random.default_rng(4)
    tokens, heads, dim = 5, 3, 16
    q, weight = rng.standard_normal((tokens, heads, dim)).astype(np.float32), rng.uniform(0.5, 1.5, size=dim)
    before = rng.standard_normal((40, 64)).astype(np.float32)
    pool, out = upload(runtime, before), empty(runtime, q.size)
    rot = {"base": 100.0, "dims": 8}
    run(runtime, "llmopt_row_attention_prepare_f32",
        [upload(runtime, q), upload(runtime, weight), upload(runtime, weight), upload(runtime, rotary_pairs(32, RotarySpec(8, 100.0))), out,
         pool, upload(runtime, np.arange(32, dtype=np.uint32)[None]), upload(runtime, np.array([7], np.uint32)),
         upload(runtime, np.array([0], np.uint32))],
        parameters.row_attention_prepare(
            sequences=1, tokens=tokens, heads=heads, kv_heads=1, dim=dim, vdim=16, stride=heads * dim, q_column=0, k_column=0, v_column=0,
            rotary_dims=8, trig_rows=32, token_stride=64, key_offset=0, value_offset=16, table_stride=32, table_rows=1, pool_rows=40,
            head_norm=True, epsilon=1e-5, own_keys=False))
    close(download(out, q.shape), plain.rotate(plain.rms(q.astype(np.float64), 1e-5) * weight, np.arange(7, 12), rot), 3e-6)
    assert np.array_equal(download(pool, before.shape), before)


# ---- experts -------------------------------------------------------------------------------------------

EXPERTS = [  # rows, experts, top, width, inner
    (1, 5, 2, 104, 48), (1, 1, 1, 64, 16), (2, 40, 3, 96, 24), (8, 16, 16, 128, 64), (9, 300, 8, 64, 8), (33, 12, 1, 192, 96),
    (64, 1000, 2, 40, 16), (64, 7, 2, 256, 40), (17, 64, 4, 1024, 264), (3, 7, 2, 51, 31), (65, 9, 2, 104, 72), (150, 40, 3, 96, 24),
    (700, 6, 2, 128, 64), (130, 3, 3, 50, 17), (300, 200, 1, 64, 32), (1000, 4, 1, 256, 136)]


def expert_weights(rng, experts, width, inner):
    gate, up = (bf16_round(rng.standard_normal((experts, inner, width)) / np.sqrt(width)) for _ in range(2))
    down = bf16_round(rng.standard_normal((experts, width, inner)) / np.sqrt(inner))
    return gate, up, down


@pytest.mark.parametrize("rows,experts,top,width,inner", EXPERTS)
def test_routes(runtime, rows, experts, top, width, inner):
    """Choices in the order of their scores, the lower index first among equals, in both forms; the plan lists every
    pair once, sorted by expert and in order."""
    from llmopt_b200 import parameters

    rng = np.random.default_rng(rows + experts)
    logits = rng.standard_normal((rows, experts)).astype(np.float32) * 3
    logits[:, ::3] = np.round(logits[:, ::3])  # equals
    logits[0] = 1.0
    size = dict(rows=rows, experts=experts, top=top)
    want = plain.chosen_experts(logits, top)
    scores = plain.sigmoid(np.take_along_axis(logits.astype(np.float64), want, 1))
    z, pairs = upload(runtime, logits), rows * top
    chosen, weight, row_of, score_of, slot_of = (upload(runtime, np.zeros(max(pairs, 4), np.uint32)) for _ in range(5))
    most = pairs // 128 + min(experts, pairs)
    plan = upload(runtime, np.zeros(4 * (1 + most), np.uint32))
    run(runtime, "llmopt_route_rows_f32", [z, chosen, weight], parameters.route(**size))
    assert np.array_equal(chosen.to_numpy(np.uint32)[:pairs].reshape(rows, top), want)
    close(download(weight, (rows, top)), scores, 1e-6)
    run(runtime, "llmopt_route_plan", [chosen, weight, plan, row_of, score_of, slot_of], parameters.route(**size))
    order = np.argsort(want.reshape(-1), kind="stable")
    assert np.array_equal(row_of.to_numpy(np.uint32)[:pairs], order // top)
    close(download(score_of, (pairs,)), scores.reshape(-1)[order], 1e-6)
    assert np.array_equal(np.argsort(order), slot_of.to_numpy(np.uint32)[:pairs])
    counts = np.bincount(want.reshape(-1), minlength=experts)
    tiles = [(e, first, min(first + 128, end)) for e, (begin, end) in enumerate(zip(np.cumsum(counts) - counts, np.cumsum(counts)))
             for first in range(begin, end, 128)]
    entries = plan.to_numpy(np.uint32).reshape(-1, 4)
    assert entries[0, 0] == len(tiles) <= most and np.array_equal(entries[1:1 + len(tiles), :3], np.array(tiles, np.uint32))
    if rows > 64:
        return
    from llmopt_b200.feed_forward import route_words

    route = upload(runtime, np.full(route_words(rows, experts, top), 0x7FC00000, np.uint32))
    run(runtime, "llmopt_route_step_f32", [z, route], parameters.route(**size))
    words, used = route.to_numpy(np.uint32), np.nonzero(counts)[0]
    first_at = 4 + (experts + 3) // 4 * 4
    row_at = first_at + (experts + 4) // 4 * 4
    score_at = row_at + pairs
    assert words[0] == len(used) and np.array_equal(words[4:4 + len(used)], used)
    assert np.array_equal(words[first_at:first_at + len(used) + 1], np.concatenate([[0], np.cumsum(counts[used])]))
    assert np.array_equal(words[row_at:row_at + pairs], order // top)
    close(words[score_at:score_at + pairs].view(np.float32), scores.reshape(-1)[order], 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,top,width,inner", EXPERTS)
def test_experts(runtime, dtype, rows, experts, top, width, inner):
    """The whole sublayer through its record builder, against expert(score * input) summed over the choices."""
    from llmopt_b200.feed_forward import RoutedExperts
    from llmopt_b200.mixers import Step
    from llmopt_b200.model import ExpertsSpec
    from llmopt_b200 import parameters

    rng = np.random.default_rng(rows * 7 + experts)
    if experts > 100 and dtype == "float32":
        inner = min(inner, 16)
    x = bf16_round(rng.standard_normal((rows, width)))
    gate, up, down = expert_weights(rng, experts, width, inner)
    # clear choices: the router reads marks that rows carry for their experts
    router = rng.standard_normal((experts, width)) / np.sqrt(width)
    weights = {"m.router": bf16_round(router * 2)}
    for e in range(experts):
        weights |= {f"m.e{e}.gate": gate[e], f"m.e{e}.up": up[e], f"m.e{e}.down": down[e]}
    margins = []
    for _ in range(200):
        margins.clear()
        plain.routed_experts(x.astype(np.float64), weights, "m", {"experts": experts, "top": top}, margins)
        close_calls = np.nonzero(margins[0] < 2e-3)[0] if margins else ()
        if not len(close_calls):
            break
        x[close_calls] = bf16_round(rng.standard_normal((len(close_calls), width)))
    want_sum = plain.routed_experts(x.astype(np.float64), weights, "m", {"experts": experts, "top": top})
    (post, post_norm), (after, next_norm) = norm_vector(rng, width), norm_vector(rng, width)
    residual = rng.standard_normal((rows, width))

    class Engine:
        itemsize, suffix_, max_rows = (2 if dtype == "bfloat16" else 4), suffix(dtype), rows
        config = type("Config", (), {"width": width})

        def __init__(self):
            self.suffix = suffix(dtype)

        def upload_matrix(self, array):
            return upload(runtime, np.asarray(array), dtype)

        def work32(self, name, columns):
            return empty(runtime, rows * columns)

        def scratch(self, name, nbytes):
            return upload(runtime, np.full((nbytes + 3) // 4 + 4, 0x7FC00000, np.uint32))  # NaN: nothing unwritten may be read

        def record_linear(self, step, x, weight, out, *, m, n, k, split, out32):
            run(runtime, step.element("dense_linear"), [x, weight, weight, out32, out32, weight, weight],
                parameters.dense_linear(m=m, n=n, k=k, split=split))

    engine = Engine()
    step = Step(engine, 1, rows, None, None, None, lambda *a: run(runtime, *a))
    kept, out = upload(runtime, residual), empty(runtime, rows * width, dtype)

    class Stream:
        x = None
        ending = [upload(runtime, post), upload(runtime, after), kept, out]

    step.stream = Stream()
    step.stream.x = upload(runtime, x, dtype)
    RoutedExperts(engine, ExpertsSpec(experts=experts, top=top, width=inner), weights, "m").record(step)
    want = residual.astype(np.float32) + post_norm(want_sum)
    close(download(kept, (rows, width)), want, 1e-2 if dtype == "bfloat16" else 3e-6, "residual")
    close(download(out, (rows, width), dtype), next_norm(want), 1.5e-2 if dtype == "bfloat16" else 3e-6, "next input")


def test_experts_refuse_what_does_not_fit(runtime):
    from llmopt_b200 import parameters

    z = upload(runtime, np.zeros((1, 4), np.float32))
    with pytest.raises(Exception, match="choice of them"):
        run(runtime, "llmopt_route_rows_f32", [z, z, z], parameters.route(rows=1, experts=4, top=5))
    with pytest.raises(Exception, match="too short"):
        run(runtime, "llmopt_route_rows_f32", [z, z, z], parameters.route(rows=2, experts=4, top=1))
    with pytest.raises(Exception, match="too short"):
        run(runtime, "llmopt_route_step_f32", [z, z], parameters.route(rows=1, experts=4, top=4))


# ---- whole models --------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def references():
    found = {}

    def get(name, length=150, seed=7):
        key = name, length, seed
        if key not in found:
            config = SANDWICHES[name]
            weights = weights_of(config)
            found[key] = config, weights, Reference(config, weights, settled_tokens(config, weights, length, seed))
        return found[key]
    return get


CUTS = {"one prompt": [150], "portions": [2, 3, 64, 2, 31, 33, 15], "pairs and singles": [1, 2, 1, 65, 1, 1, 2, 2, 75],
        "pairs": [2] * 75, "decoding": [100] + [1] * 50, "decoding from the start": [1] * 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SANDWICHES))
def test_prompts_portions_and_decoding(runtime, references, dtype, name):
    """The same sequence as one prompt, in portions of every kind, and token by token."""
    config, weights, reference = references(name)
    engine = build(runtime, config, weights, capacity=160, sequences=2, dtype=dtype)
    for label, counts in CUTS.items():
        sequence, at = engine.open(), 0
        for count in counts:
            got = engine.run([(sequence, reference.tokens[at:at + count], list(range(count)))])[0]
            reference.check(got, np.arange(at, at + count), dtype, label)
            at += count
        engine.close(sequence)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_runs_in_portions_of_its_own(runtime, references, dtype):
    config, weights, reference = references("square", 500)
    engine = build(runtime, config, weights, capacity=512, dtype=dtype, prompt_rows=192)
    places = [0, 5, 63, 64, 127, 128, 191, 192, 193, 383, 384, 498, 499]
    got = engine.run([(engine.open(), reference.tokens, places)])[0]
    reference.check(got, places, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_side_by_side_equal_each_alone(runtime, dtype):
    config = SANDWICHES["kept"]
    weights = weights_of(config)
    rng = np.random.default_rng(9)
    lengths = [1, 7, 40, 90, 3]
    streams = [settled_tokens(config, weights, length + 30, seed=20 + i) for i, length in enumerate(lengths)]
    engine = build(runtime, config, weights, batch=5, capacity=128, dtype=dtype)
    rows = [engine.open() for _ in lengths]
    first = engine.run([(row, stream[:length], [length - 1]) for row, stream, length in zip(rows, streams, lengths)])
    together = [[logits[0]] for logits in first]
    for step in range(30):
        live = [i for i in range(5) if step < 10 * (i + 1)]  # sequences leave one after the other
        order = rng.permutation(live)
        got = engine.run([(rows[i], [streams[i][lengths[i] + step]], [0]) for i in order])
        for i, logits in zip(order, got):
            together[i].append(logits[0])
    for i, (stream, length) in enumerate(zip(streams, lengths)):
        alone = build(runtime, config, weights, capacity=128, dtype=dtype)
        sequence = alone.open()
        apart = [alone.run([(sequence, stream[:length], [length - 1])])[0][0]]
        for step in range(len(together[i]) - 1):
            apart.append(alone.run([(sequence, [stream[length + step]], [0])])[0][0])
        places = np.arange(length - 1, length - 1 + len(apart))
        Reference(config, weights, stream).check(together[i], places, dtype)
        assert np.median(logit_error(together[i], np.array(apart, np.float64))) <= (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rows_and_pages_used_again(runtime, dtype):
    """Sequences of changing lengths pass through three rows and few pages of four slots; nothing of an earlier one may
    be seen."""
    config = SANDWICHES["odd"]
    weights = weights_of(config)
    rng = np.random.default_rng(10)
    engine = build(runtime, config, weights, capacity=64, sequences=3, token_capacity=100, page=4, dtype=dtype)
    live = []
    for turn in range(14):
        length = int(rng.integers(4, 30))
        tokens = settled_tokens(config, weights, length + 2, seed=100 + turn)
        reference = Reference(config, weights, tokens)
        sequence, cut = engine.open(), int(rng.integers(1, length))
        got = [engine.run([(sequence, part, list(range(len(part))))])[0] for part in (tokens[:cut], tokens[cut:length])]
        reference.check(np.concatenate(got), np.arange(length), dtype, turn)
        live.append((sequence, reference))
        if len(live) == 3:
            sequence, reference = live.pop(int(rng.integers(0, 3)))
            at = len(reference.tokens) - 2
            got = engine.run([(sequence, reference.tokens[at:], [0, 1])])[0]
            reference.check(got, [at, at + 1], dtype, turn)
            engine.close(sequence)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(runtime, dtype):
    config = sandwich_config([window_layer(size=50, keep_first=4, mlp=dense_mlp(64)), window_layer(kv_from=0, size=120, keep_first=0),
                              window_layer(heads=4, kv_heads=2, dim=32, vdim=32, size=None, mlp=routed_mlp(6, 2, 40))], vocab=90)
    weights = weights_of(config, seed=4)
    tokens = settled_tokens(config, weights, 500, seed=12)
    engine = build(runtime, config, weights, capacity=512, dtype=dtype)
    sequence = engine.open()
    engine.run([(sequence, tokens[:20], [])])
    got = np.array([engine.run([(sequence, [token], [0])])[0][0] for token in tokens[20:]])
    Reference(config, weights, tokens).check(got, np.arange(20, 500), dtype)


def test_a_marked_token_is_seen_exactly_inside_the_windows(runtime):
    """One token of the context is exchanged; with one layer of attention the logits of a later place move exactly when
    that place sees it, in a prompt and in decoding."""
    size, keep = 20, 3
    config = sandwich_config([window_layer(size=size, keep_first=keep, mlp=dense_mlp(48))], width=64, vocab=90)
    weights = weights_of(config, seed=5)
    base = np.random.default_rng(3).integers(0, 89, size=80).tolist()
    engine = build(runtime, config, weights, capacity=96, dtype="float32")

    def logits(tokens, prompt):
        sequence = engine.open()
        rows = [engine.run([(sequence, tokens[:prompt], list(range(prompt)))])[0]]
        rows += [engine.run([(sequence, [token], [0])])[0] for token in tokens[prompt:]]
        engine.close(sequence)
        return np.concatenate(rows)

    for prompt in (80, 30):
        before = logits(base, prompt)
        for place in (0, keep - 1, keep, 15, 16, 31):
            moved = np.max(np.abs(logits(base[:place] + [89] + base[place + 1:], prompt) - before), axis=1) > 1e-4
            sees = [t >= place and (t - place < size or place < keep) for t in range(80)]
            assert moved.tolist() == sees, (prompt, place)


def test_greedy_generation_through_the_engine(runtime):
    """More prompts than places in the batch, unequal lengths: the tokens of the plain restatement."""
    config = SANDWICHES["kept"]
    weights = weights_of(config, seed=3)
    rng = np.random.default_rng(11)
    prompts = [rng.integers(0, config["vocab"], size=n).tolist() for n in (5, 1, 33, 12, 2)]
    wanted = [greedy(config, weights, prompt, 16) for prompt in prompts]
    assert min(gap for _, gap in wanted) > 1e-4
    engine = build(runtime, config, weights, batch=2, capacity=64, dtype="float32")
    assert engine.generate(prompts, 16) == [tokens for tokens, _ in wanted]
    batch = build(runtime, config, weights, batch=2, capacity=64, dtype="float32")
    pair = [prompts[0], prompts[0][::-1]]
    second = greedy(config, weights, pair[1], 16)[0]
    stream = [[batch.prefill(prompt, sequence) for sequence, prompt in enumerate(pair)]]
    for step in range(8):
        stream.append(batch.step(stream[-1], 5 + step))
    assert [t[0] for t in stream] == wanted[0][0][:9] and [t[1] for t in stream] == second[:9]
    chained, elapsed = batch.generate_chained(stream[-1], 13, 7)
    assert chained == wanted[0][0][9:16] and elapsed > 0
    draws = [engine.generate(prompts[:2], 8, temperature=1.0, top_k=20, seed=s) for s in (5, 5, 6)]
    assert draws[0] == draws[1] != draws[2]


def checkpoint(folder, config, weights):
    from llmopt_b200.safetensors_archive import as_bfloat16_bits

    (folder / "config.json").write_text(json.dumps(config))
    write_checkpoint(folder / "model.safetensors", {name: ("BF16", as_bfloat16_bits(value)) for name, value in weights.items()})


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(runtime, references, tmp_path, dtype):
    """The program end to end: a checkpoint on disk, steps on standard input, logits in files."""
    config, weights, reference = references("kept")
    checkpoint(tmp_path, config, weights)
    tokens = reference.tokens
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[18:90], "want": [1, 71]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": tokens[90:91], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": tokens[:1], "want": [0]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    out.mkdir()
    done = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype,
                           "--out", str(out), "--max-tokens", "91"], input="".join(json.dumps(s) + "\n" for s in steps),
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
    for step, places in ((0, [0, 16]), (2, [19, 89]), (3, [90]), (4, [0])):
        reference.check(np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, config["vocab"]), places, dtype, step)
    assert not (out / "1.f32").exists()


def test_generate_command(runtime, tmp_path, capsys):
    from llmopt_b200 import generate

    config = SANDWICHES["kept"]
    weights = weights_of(config, seed=3)
    checkpoint(tmp_path, config, weights)
    generate.main(["--model", str(tmp_path), "--prompt", "3,99,41", "--prompt", "7", "--tokens", "6", "--dtype", "float32"])
    wanted = [greedy(config, weights, prompt, 6)[0] for prompt in ([3, 99, 41], [7])]
    assert capsys.readouterr().out.splitlines() == [",".join(map(str, tokens)) for tokens in wanted]

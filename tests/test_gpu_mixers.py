"""The sequence-mixer kernels, cache, states and engine on the GPU against the plain restatement of the
equations (``oracle_mixers``): each mechanism alone, then whole models in prompts, portions and decoding."""

import numpy as np
import pytest

import oracle_mixers as plain
from mixer_models import MODELS, bf16_round, config_of, memory_layer, parallel_layer, weights_of

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")


def suffix(dtype):
    return "f32" if dtype == "float32" else "bf16"


def upload(runtime, array, dtype="float32"):
    from llmopt_b200.cuda_native import Buffer
    from llmopt_b200.safetensors_archive import as_bfloat16_bits

    array = np.ascontiguousarray(array)
    if dtype == "bfloat16":
        array = as_bfloat16_bits(array.astype(np.float32))
    elif array.dtype == np.float64:
        array = array.astype(np.float32)
    return Buffer.of_array(runtime, array)


def empty(runtime, elements, dtype="float32"):
    from llmopt_b200.cuda_native import Buffer

    return Buffer.create(runtime, max(elements * (2 if dtype == "bfloat16" else 4), 16))


def download(buffer, shape, dtype="float32"):
    count = int(np.prod(shape))
    if dtype == "bfloat16":
        return (buffer.to_numpy(np.uint16)[:count].astype(np.uint32) << 16).view(np.float32).reshape(shape)
    return buffer.to_numpy(np.float32)[:count].reshape(shape)


def close(actual, expected, tolerance, label=""):
    actual, expected = np.asarray(actual, np.float64), np.asarray(expected, np.float64)
    assert actual.shape == expected.shape and np.all(np.isfinite(actual)), label
    scale = max(np.max(np.abs(expected)), 1e-6)
    error = np.max(np.abs(actual - expected)) / scale
    assert error <= tolerance, f"{label}: {error:.3e} of the scale exceeds {tolerance:.1e}"


# ---- mechanisms alone ----------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k,split", [
    (1, 24, 104, 24), (1, 300, 64, 256), (3, 77, 50, 40), (8, 130, 200, 130), (9, 64, 72, 0), (17, 40, 1000, 33),
    (33, 96, 128, 64), (64, 333, 264, 100), (65, 80, 104, 72), (130, 200, 256, 128), (257, 520, 336, 512), (300, 61, 50, 30),
    (140, 1000, 1024, 0), (200, 19000, 64, 19000), (1, 16, 4096, 16), (40, 4096, 16, 0)])
def test_dense_linear(runtime, dtype, m, n, k, split):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(m * 1000 + n)
    x, w = bf16_round(rng.standard_normal((m, k))), bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    bias = rng.standard_normal(n).astype(np.float32)
    table, ids = bf16_round(rng.standard_normal((20, n + 7))), rng.integers(0, 20, size=m)
    y = x.astype(np.float64) @ w.T.astype(np.float64)
    buffers = [upload(runtime, x, dtype), upload(runtime, w, dtype), upload(runtime, bias), empty(runtime, m * max(split, 1), dtype),
               empty(runtime, m * max(n - split, 1)), upload(runtime, ids.astype(np.int64)), upload(runtime, table, dtype)]
    for epilogue, has_bias, want in ((None, True, y + bias), (None, False, y), ("gelu", False, plain.gelu_erf(y)),
                                     ("token_gate", True, plain.gelu_tanh(y + bias) * table[ids][:, 5:5 + n])):
        runtime.dispatch("llmopt_dense_linear_" + suffix(dtype), buffers=buffers, parameters=parameters.dense_linear(
            m=m, n=n, k=k, split=split, has_bias=has_bias, epilogue=epilogue, table_rows=20, table_stride=n + 7, table_offset=5))
        if split:
            close(download(buffers[3], (m, split), dtype), want[:, :split], 6e-3 if dtype == "bfloat16" else 3e-6, epilogue)
        if split < n:
            close(download(buffers[4], (m, n - split)), want[:, split:], 1e-5, epilogue)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [97, 104, 192, 1028, 4096, 8192, 9000])
def test_residual_norm(runtime, dtype, width):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(width)
    rows, eps = 5, 0.01
    x, y, y2 = (rng.standard_normal((rows, width)) * s for s in (1.0, 3.0, 0.01))
    w, wl, wr = (rng.uniform(-1, 2, size=width) for _ in range(3))
    buffers = [upload(runtime, v) for v in (x, y, w, y2, wl, wr)] + [empty(runtime, rows * width), empty(runtime, rows * width, dtype)]
    mean = 0.5 * (plain.rms(y, eps) * wl + plain.rms(y2, eps) * wr)
    for pair, offset, value in ((False, 1.0, y), (False, 0.0, y), (True, 1.0, mean), (True, 0.0, mean)):
        runtime.dispatch("llmopt_residual_norm_" + suffix(dtype), buffers=buffers, parameters=parameters.residual_norm(
            rows=rows, width=width, epsilon=eps, weight_offset=offset, pair=pair))
        want = x + plain.rms(value, eps) * (offset + w)
        close(download(buffers[6], (rows, width)), want, 2e-6, (pair, offset))
        if dtype == "bfloat16":
            close(download(buffers[7], (rows, width), dtype), want, 5e-3)


def test_gather_norm_and_greedy_pick(runtime):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(0)
    x, w = rng.standard_normal((7, 150)), rng.standard_normal(150)
    chosen = np.array([6, 0, 3, 3], np.uint32)
    for dtype in DTYPES:
        out = empty(runtime, 4 * 150, dtype)
        runtime.dispatch("llmopt_gather_norm_" + suffix(dtype), buffers=[upload(runtime, x), upload(runtime, chosen), upload(runtime, w), out],
                         parameters=parameters.gather_norm(count=4, source_rows=7, width=150, epsilon=1e-5, weight_offset=1.0))
        close(download(out, (4, 150), dtype), (plain.rms(x, 1e-5) * (1 + w))[chosen], 5e-3 if dtype == "bfloat16" else 2e-6)
    for columns in (1, 31, 5000):
        logits = rng.standard_normal((3, columns)).astype(np.float32)
        logits[1, :] = -2.0
        logits[1, columns // 2:] = -1.0  # the first of equals wins
        best, picked, ids, past = (upload(runtime, np.zeros(3 * 8, np.int64)), upload(runtime, np.zeros(4, np.int32)),
                                   upload(runtime, np.zeros(3, np.int64)), upload(runtime, np.array([4, 5, 6], np.uint32)))
        runtime.dispatch("llmopt_argmax_f32", buffers=[upload(runtime, logits), best], parameters=parameters.u32s([3, columns, 8]))
        runtime.dispatch("llmopt_advance_tokens", buffers=[best, picked, ids, past], parameters=parameters.u32s([3, 8, 1]))
        want = np.argmax(logits, axis=1).tolist()
        assert picked.to_numpy(np.int32)[:3].tolist() == want and ids.to_numpy(np.int64).tolist() == want
        assert past.to_numpy(np.uint32).tolist() == [5, 6, 7]


class AttentionBench:
    """The two attention kernels over one layer's cache with scattered slots."""

    def __init__(self, runtime, dtype, *, heads, kv_heads, dim, vdim, rot, scale, sink=True, capacity=2100, head_norm=True, seed=0):
        from llmopt_b200.bizodra import _rotary
        from llmopt_b200.kv_cache import RowLayout
        from llmopt_b200.quantize import rotary_pairs

        self.runtime, self.dtype, self.size = runtime, dtype, dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        self.rot, self.scale, self.sink, self.capacity, self.head_norm = rot, scale, sink, capacity, head_norm
        rng = np.random.default_rng(seed)
        self.layout = RowLayout([(1, 8, 8), (kv_heads, dim, vdim), (2, 16, 8)])  # the layer in the middle
        self.slots = capacity + 40
        self.pool = empty(runtime, self.slots * self.layout.token_elements, dtype)
        self.order = rng.permutation(self.slots)[:capacity].astype(np.uint32)
        table = np.zeros((3, capacity), np.uint32)
        table[1] = self.order
        self.table, self.row = upload(runtime, table), upload(runtime, np.array([1], np.uint32))
        self.trig = upload(runtime, rotary_pairs(capacity, _rotary(rot)))
        self.norms = [rng.uniform(0.5, 1.5, size=dim) for _ in range(2)]
        self.norm_buffers = [upload(runtime, w) for w in self.norms]
        self.past = 0
        self.eps = 1e-5

    def run(self, q, k, v, splits):
        """Appends tokens; returns their read-outs."""
        from llmopt_b200 import parameters

        tokens, size = q.shape[0], self.size
        stride = size["heads"] * size["dim"] + size["kv_heads"] * (size["dim"] + size["vdim"]) + 3
        projected = np.concatenate([v.reshape(tokens, -1), np.zeros((tokens, 3)), q.reshape(tokens, -1), k.reshape(tokens, -1)], axis=1)
        v_columns = size["kv_heads"] * size["vdim"]
        query, out = empty(self.runtime, q.size, self.dtype), empty(self.runtime, tokens * size["heads"] * size["vdim"], self.dtype)
        past = upload(self.runtime, np.array([self.past], np.uint32))
        region = self.layout.regions[1]
        cache = dict(token_stride=self.layout.token_elements, key_offset=region.key_offset, value_offset=region.value_offset,
                     table_stride=self.capacity, table_rows=3, pool_rows=self.slots)
        self.runtime.dispatch(
            "llmopt_row_attention_prepare_" + suffix(self.dtype),
            buffers=[upload(self.runtime, projected, self.dtype), *self.norm_buffers, self.trig, query, self.pool, self.table, past, self.row],
            parameters=parameters.row_attention_prepare(
                sequences=1, tokens=tokens, **size, stride=stride, q_column=v_columns + 3,
                k_column=v_columns + 3 + size["heads"] * size["dim"], v_column=0, rotary_dims=self.rot["dims"],
                trig_rows=self.capacity, **cache, head_norm=self.head_norm, epsilon=self.eps))
        scratch = empty(self.runtime, 64 + size["kv_heads"] * splits * (32 + 16 * 256))
        for _ in range(2):  # the arrival counters return to zero
            self.runtime.dispatch(
                "llmopt_row_attention_" + suffix(self.dtype),
                buffers=[query, self.pool, self.table, past, self.row, out, scratch, query],
                parameters=parameters.row_attention(sequences=1, tokens=tokens, **size, **cache, sink=self.sink, splits=splits, scale=self.scale))
        self.past += tokens
        return download(out, (tokens, size["heads"], size["vdim"]), self.dtype)

    def expected(self, q, k, v):
        positions = np.arange(q.shape[0])
        if self.head_norm:
            q, k = plain.rms(q, self.eps) * self.norms[0], plain.rms(k, self.eps) * self.norms[1]
        q, k = plain.rotate(q.astype(np.float64), positions, self.rot), plain.rotate(k.astype(np.float64), positions, self.rot)
        if self.sink:
            return plain.sink_attention(q, k, v, self.scale)
        group, out = q.shape[1] // k.shape[1], np.zeros((*q.shape[:2], v.shape[2]))
        for h in range(q.shape[1]):
            score = np.where(np.tril(np.ones((len(q), len(q)), bool)), (q[:, h] @ k[:, h // group].T) * self.scale, -np.inf)
            weight = np.exp(score - score.max(axis=1, keepdims=True))
            out[:, h] = weight / weight.sum(axis=1, keepdims=True) @ v[:, h // group]
        return out


ATTENTION = {
    "gqa": dict(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.3, rot={"base": 5000.0, "dims": 16, "scaling": {
        "factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}}),
    "square64": dict(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, rot={"base": 10000.0, "dims": 64}),
    "square128": dict(heads=8, kv_heads=1, dim=128, vdim=128, scale=0.09, rot={"base": 1e5, "dims": 32}),
    "wide": dict(heads=2, kv_heads=2, dim=72, vdim=200, scale=0.1, rot={"base": 100.0, "dims": 72}),
    "narrow": dict(heads=16, kv_heads=1, dim=48, vdim=32, scale=0.2, rot={"base": 1e4, "dims": 48}),
    "odd": dict(heads=9, kv_heads=3, dim=18, vdim=10, scale=0.5, rot={"base": 1e6, "dims": 4}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ATTENTION))
def test_attention_in_portions(runtime, dtype, name):
    """Portions down to one token over scattered slots, split over the keys or not."""
    size = ATTENTION[name]
    rng = np.random.default_rng(3)
    bench = AttentionBench(runtime, dtype, **size)
    counts = [1, 2, 70, 3, 64, 1, 1, 130, 2, 5, 1]
    total = sum(counts)
    q, k, v = (bf16_round(rng.standard_normal((total, h, d))) for h, d in (
        (size["heads"], size["dim"]), (size["kv_heads"], size["dim"]), (size["kv_heads"], size["vdim"])))
    want, at = bench.expected(q, k, v), 0
    for index, count in enumerate(counts):
        got = bench.run(q[at:at + count], k[at:at + count], v[at:at + count], splits=[1, 7, 33][index % 3])
        close(got, want[at:at + count], 1.5e-2 if dtype == "bfloat16" else 3e-6, f"portion {index}")
        at += count


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_finds_one_far_key(runtime, dtype):
    """Among 2000 keys one stands out for the last tokens; in a prompt, in a portion and alone, at the first
    position, at the borders of the kernels' key tiles and splits, and for the token itself."""
    size = dict(heads=2, kv_heads=1, dim=64, vdim=32)
    rng = np.random.default_rng(5)
    total = 2005
    for place in (0, 1, 15, 16, 63, 64, 65, 127, 1023, 1024, 1999, 2000, 2004):
        q, k = (bf16_round(0.2 * rng.standard_normal((total, h, 64))) for h in (2, 1))
        v = bf16_round(rng.standard_normal((total, 1, 32)))
        mark = rng.standard_normal(64)
        k[place, 0] = bf16_round(mark)
        q[2000:, :] = bf16_round(mark)
        bench = AttentionBench(runtime, dtype, **size, rot={"base": 1e4, "dims": 2}, scale=0.25, head_norm=False)
        want = bench.expected(q, k, v)
        bench.run(q[:1900], k[:1900], v[:1900], 1)
        got = np.concatenate([bench.run(q[a:b], k[a:b], v[a:b], s) for a, b, s in
                              ((1900, 2001, 1), (2001, 2003, 40), (2003, 2004, 64), (2004, 2005, 9))])
        close(got, want[1900:], 1.5e-2 if dtype == "bfloat16" else 1e-4, f"key {place}")
        seen = [t for t in range(2000, total) if t >= place]
        assert seen and all(np.argmax(np.abs(want[t, 0] @ v[:, 0].T)) == place for t in seen[-1:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 20, 90])
def test_attention_sink(runtime, dtype, tokens):
    """With all scores far below zero the sink takes nearly everything; without it nothing is lost."""
    size = dict(heads=2, kv_heads=1, dim=32, vdim=32, rot={"base": 1e4, "dims": 2}, scale=1.0, head_norm=False)
    rng = np.random.default_rng(tokens)
    q = bf16_round(np.abs(rng.standard_normal((tokens, 2, 32))) * 0.3)
    k = bf16_round(-np.abs(rng.standard_normal((tokens, 1, 32))) * 0.5)
    v = bf16_round(1.0 + rng.random((tokens, 1, 32)))
    for sink in (True, False):
        for splits in (1, 5):
            bench = AttentionBench(runtime, dtype, **size, sink=sink)
            want, got = bench.expected(q, k, v), bench.run(q, k, v, splits)
            close(got, want, 1.5e-2 if dtype == "bfloat16" else 3e-6, (sink, splits))
        assert (want[0].max() < 0.5) == sink


def delta_inputs(rng, tokens, heads, kv_heads, dim, vdim, taps):
    qk, vs = kv_heads * dim, heads * vdim
    raw = bf16_round(rng.standard_normal((tokens, 2 * qk + vs)))
    conv = (rng.standard_normal((2 * qk + vs, taps)) * 0.6).astype(np.float32)
    scalars = rng.standard_normal((tokens, 2 * heads)).astype(np.float32)
    a_log, dt_bias = np.log(rng.uniform(0.5, 4.0, size=heads)), rng.uniform(-4.0, 0.0, size=heads)
    return raw, conv, scalars, a_log, dt_bias


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(4, 2, 36, 44, 3), (3, 3, 104, 16, 2), (6, 1, 10, 33, 5),
                                                          (2, 1, 128, 128, 4), (2, 2, 250, 70, 1), (1, 1, 180, 32, 9)])
def test_gated_delta_rule(runtime, dtype, heads, kv_heads, dim, vdim, taps):
    """Convolution, unit vectors, gates and the state, in portions (also shorter than the convolution)."""
    from llmopt_b200 import parameters
    from llmopt_b200.kv_cache import matrix_state_elements

    rng = np.random.default_rng(dim)
    counts = [1, 2, 40, 3, 33, 1, 32, 1, 70]
    tokens = sum(counts)
    raw, conv, scalars, a_log, dt_bias = delta_inputs(rng, tokens, heads, kv_heads, dim, vdim, taps)
    qk, vs = kv_heads * dim, heads * vdim
    filtered = plain.short_conv(raw.astype(np.float64), conv)
    which = np.arange(heads) // (heads // kv_heads)
    q = plain.unit(filtered[:, :qk].reshape(tokens, kv_heads, dim)) * dim ** -0.5
    k = plain.unit(filtered[:, qk:2 * qk].reshape(tokens, kv_heads, dim))
    v = filtered[:, 2 * qk:].reshape(tokens, heads, vdim)
    beta = plain.sigmoid(scalars[:, :heads].astype(np.float64))
    decay = np.exp(-np.exp(a_log) * plain.softplus(scalars[:, heads:] + dt_bias))
    want, state = plain.delta_scan(q[:, which], k[:, which], v, decay, beta)

    rows, stride = 3, matrix_state_elements(heads, dim, vdim, normalized=False)
    # what an earlier sequence left in the row must not matter
    pool = upload(runtime, rng.standard_normal((rows, stride)))
    kept = upload(runtime, rng.standard_normal((rows, (2 * qk + vs) * taps)), dtype)
    weights = [upload(runtime, x) for x in (conv, a_log, dt_bias)]
    row, at, got = upload(runtime, np.array([2], np.uint32)), 0, []
    for count in counts:
        part = slice(at, at + count)
        past = upload(runtime, np.array([at], np.uint32))
        projected, extra = upload(runtime, raw[part], dtype), upload(runtime, scalars[part])
        out = [empty(runtime, count * n) for n in (qk, qk, vs, heads, heads, vs)]
        prepare = parameters.delta_prepare(
            sequences=1, tokens=count, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, taps=taps, stride=2 * qk + vs, q_column=0,
            k_column=qk, v_column=2 * qk, scalar_stride=2 * heads, beta_column=0, decay_column=heads, state_rows=rows)
        runtime.dispatch("llmopt_delta_prepare_" + suffix(dtype),
                         buffers=[projected, extra, weights[0], kept, past, row, weights[1], weights[2], *out[:5]], parameters=prepare)
        runtime.dispatch("llmopt_conv_state_" + suffix(dtype), buffers=[projected, kept, past, row], parameters=prepare)
        runtime.dispatch("llmopt_delta_scan_f32", buffers=[*out[:5], pool, past, row, out[5]], parameters=parameters.state_scan(
            sequences=1, tokens=count, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, q_stride=qk, q_column=0, k_stride=qk,
            k_column=0, v_stride=vs, v_column=0, scalar_stride=heads, first_column=0, second_column=0, state_rows=rows,
            state_stride=stride))
        got.append(download(out[5], (count, heads, vdim)))
        close(download(out[0], (count, kv_heads, dim)), q[part], 3e-6, "unit q")
        close(download(out[3], (count, heads)), decay[part], 2e-6, "decay")
        at += count
    close(np.concatenate(got), want, 2e-5, "read-out")
    final = download(pool, (rows, stride))[2][:heads * vdim * dim].reshape(heads, vdim, dim).transpose(0, 2, 1)
    close(final, state, 2e-5, "state")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,cap,loud", [(3, 40, 24, 6.0, 1.0), (1, 136, 40, 20.0, 8.0), (5, 7, 9, 1.0, 1.0),
                                                     (2, 64, 128, 15.0, 5.0), (2, 256, 70, 15.0, 30.0), (4, 96, 33, 3.0, 1.0)])
def test_matrix_memory(runtime, dtype, heads, dim, vdim, cap, loud):
    """Portions of several sizes; also gates that span their whole range, so that the running maximum rises
    and falls, and quiet starts, where exp(-m) bounds the denominator."""
    from llmopt_b200 import parameters
    from llmopt_b200.kv_cache import MATRIX_STATE_SLICE, matrix_state_elements

    rng = np.random.default_rng(vdim)
    counts = [1, 2, 33, 1, 40, 32, 3, 1, 65]
    tokens = sum(counts)
    raw = bf16_round(rng.standard_normal((tokens, heads * (2 * dim + vdim))) * 0.7)
    scalars = (rng.standard_normal((tokens, 2 * heads)) * loud + np.repeat([-1.0, 3.0], heads)).astype(np.float32)
    scalars[:4, :heads] -= 4.0
    qk = heads * dim
    q = raw[:, :qk].reshape(tokens, heads, dim).astype(np.float64) * dim ** -0.5
    k, v = raw[:, qk:2 * qk].reshape(tokens, heads, dim).astype(np.float64), raw[:, 2 * qk:].reshape(tokens, heads, vdim).astype(np.float64)
    log_input = cap * np.tanh(scalars[:, :heads].astype(np.float64) / cap)
    log_forget = plain.log_sigmoid(cap * np.tanh(scalars[:, heads:].astype(np.float64) / cap))
    want, (memory, norm, top) = plain.matrix_memory_scan(q, k, v, log_input, log_forget)
    # where n . q nearly cancels, the quotient amplifies rounding: compare in units of what it divides
    rows, stride = 2, matrix_state_elements(heads, dim, vdim, normalized=True)
    pool, row, at, got = upload(runtime, rng.standard_normal((rows, stride))), upload(runtime, np.array([1], np.uint32)), 0, []
    for count in counts:
        part = slice(at, at + count)
        projected, extra = upload(runtime, raw[part], dtype), upload(runtime, scalars[part])
        out, past = empty(runtime, count * heads * vdim), upload(runtime, np.array([at], np.uint32))
        width = raw.shape[1]
        runtime.dispatch("llmopt_memory_scan_" + suffix(dtype),
                         buffers=[projected, projected, projected, extra, extra, pool, past, row, out],
                         parameters=parameters.state_scan(
                             sequences=1, tokens=count, heads=heads, kv_heads=heads, dim=dim, vdim=vdim, q_stride=width, q_column=0,
                             k_stride=width, k_column=qk, v_stride=width, v_column=2 * qk, scalar_stride=2 * heads, first_column=0,
                             second_column=heads, state_rows=rows, state_stride=stride, gate_cap=cap))
        got.append(download(out, (count, heads, vdim)))
        at += count
    close(np.concatenate(got), want, 1e-4, "read-out")
    final = download(pool, (rows, stride))[1]
    close(final[:heads * vdim * dim].reshape(heads, vdim, dim).transpose(0, 2, 1), memory, 3e-5, "memory")
    slices = -(-vdim // MATRIX_STATE_SLICE)
    norms = final[heads * vdim * dim:heads * (vdim + slices) * dim].reshape(heads, slices, dim)
    tops = final[heads * (vdim + slices) * dim:][:heads * slices].reshape(heads, slices)
    for one in range(slices):
        close(norms[:, one], norm, 3e-5, "n")
        close(tops[:, one], top, 1e-5, "m")


@pytest.mark.parametrize("dtype", DTYPES)
def test_head_norm_gate(runtime, dtype):
    from llmopt_b200 import parameters

    rng = np.random.default_rng(0)
    rows, heads, dim, eps = 5, 3, 44, 1e-3
    o, gate = rng.standard_normal((rows, heads, dim)) * 2, bf16_round(rng.standard_normal((rows, heads * dim + 9)))
    for per_head, gated in ((True, plain.sigmoid), (False, plain.silu)):
        weight = rng.standard_normal(heads * dim if per_head else dim)
        out = empty(runtime, rows * heads * dim, dtype)
        runtime.dispatch("llmopt_head_norm_gate_" + suffix(dtype),
                         buffers=[upload(runtime, o), upload(runtime, gate, dtype), upload(runtime, weight), out],
                         parameters=parameters.head_norm_gate(rows=rows, heads=heads, dim=dim, gate_stride=heads * dim + 9, gate_column=9,
                                                              weight_per_head=per_head, gate_sigmoid=gated is plain.sigmoid, epsilon=eps))
        shaped = weight.reshape(heads, dim) if per_head else weight
        want = plain.rms(o, eps) * shaped * gated(gate[:, 9:].astype(np.float64)).reshape(rows, heads, dim)
        close(download(out, (rows, heads, dim), dtype), want, 5e-3 if dtype == "bfloat16" else 2e-6)


# ---- whole models --------------------------------------------------------------------------------------------

def build(runtime, config, weights, **options):
    from llmopt_b200.decode_engine import create_engine
    from llmopt_b200.model import parse_config

    return create_engine(runtime, parse_config(config), weights, **options)


def logit_error(got, want):
    """Root mean square over the vocabulary of the centred difference, in units of the logits' spread."""
    difference = np.asarray(got, np.float64) - want
    difference -= difference.mean(axis=-1, keepdims=True)
    return np.sqrt((difference ** 2).mean(axis=-1)) / np.sqrt(((want - want.mean(axis=-1, keepdims=True)) ** 2).mean())


RELATIVE = {"float32": 2.0 ** -23, "bfloat16": 2.0 ** -8}
FLOOR = {"float32": 1e-5, "bfloat16": 3e-2}


class Reference:
    """Logits of one sequence by the plain restatement, and how far rounding alone may move each."""

    def __init__(self, config, weights, tokens):
        self.config, self.weights, self.tokens = config, weights, list(tokens)
        self.logits = plain.forward(config, weights, tokens)
        self.rounding = {}

    def limit(self, dtype):
        if dtype not in self.rounding:
            self.rounding[dtype] = plain.rounding_error(self.config, self.weights, self.tokens, RELATIVE[dtype])
        return np.maximum(4.0 * self.rounding[dtype], FLOOR[dtype])

    def check(self, got, places, dtype, label=""):
        excess = logit_error(got, self.logits[places]) / self.limit(dtype)[places]
        worst = int(excess.argmax())
        assert excess[worst] <= 1.0, f"{label}: token {np.asarray(places)[worst]} is {excess[worst]:.2f} times its limit off"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompts_portions_and_decoding(runtime, dtype, name):
    """The same sequence as one prompt, in portions of every kind, and token by token."""
    config = MODELS[name]
    weights = weights_of(config)
    tokens = np.random.default_rng(7).integers(0, config["vocab"], size=150).tolist()
    reference = Reference(config, weights, tokens)
    engine = build(runtime, config, weights, capacity=160, sequences=2, dtype=dtype)
    cuts = {"one prompt": [150], "portions": [2, 3, 64, 2, 31, 33, 15], "pairs and singles": [1, 2, 1, 65, 1, 1, 2, 2, 75],
            "decoding": [100] + [1] * 50, "decoding from the start": [1] * 40}
    for label, counts in cuts.items():
        sequence, at = engine.open(), 0
        for count in counts:
            got = engine.run([(sequence, tokens[at:at + count], list(range(count)))])[0]
            reference.check(got, np.arange(at, at + count), dtype, label)
            at += count
        engine.close(sequence)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_runs_in_portions_of_its_own(runtime, dtype):
    config = MODELS["square"]
    weights = weights_of(config)
    tokens = np.random.default_rng(8).integers(0, config["vocab"], size=700).tolist()
    engine = build(runtime, config, weights, capacity=704, dtype=dtype, prompt_rows=192)
    places = [0, 5, 191, 192, 193, 383, 384, 575, 698, 699]
    got = engine.run([(engine.open(), tokens, places)])[0]
    Reference(config, weights, tokens).check(got, places, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_side_by_side_equal_each_alone(runtime, dtype):
    config = MODELS["mixed"]
    weights = weights_of(config)
    rng = np.random.default_rng(9)
    lengths = [1, 7, 40, 90, 3]
    streams = [rng.integers(0, config["vocab"], size=length + 30).tolist() for length in lengths]
    engine = build(runtime, config, weights, batch=5, capacity=128, dtype=dtype)
    rows = [engine.open() for _ in lengths]
    prompts = [(row, stream[:length], [length - 1]) for row, stream, length in zip(rows, streams, lengths)]
    first = engine.run(prompts[:3]) + engine.run(prompts[3:])
    together = [[rows_[0]] for rows_ in first]
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
        reference = Reference(config, weights, stream)
        reference.check(together[i], places, dtype)
        # the company changes nothing but the order of a few sums
        assert np.median(logit_error(together[i], np.array(apart, np.float64))) <= (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rows_and_pages_used_again(runtime, dtype):
    """Sequences of changing lengths pass through a table of three rows and few pages of four slots; nothing of
    an earlier one may be seen."""
    config = MODELS["odd"]
    weights = weights_of(config)
    rng = np.random.default_rng(10)
    engine = build(runtime, config, weights, capacity=64, sequences=3, token_capacity=100, page=4, dtype=dtype)
    live = []
    for turn in range(14):
        length = int(rng.integers(2, 30))
        tokens = rng.integers(0, config["vocab"], size=length).tolist()
        sequence = engine.open()
        cut = int(rng.integers(1, length)) if length > 1 else 0
        got = [engine.run([(sequence, part, list(range(len(part))))])[0] for part in (tokens[:cut], tokens[cut:]) if part]
        Reference(config, weights, tokens).check(np.concatenate(got), np.arange(length), dtype, turn)
        live.append((sequence, tokens))
        if len(live) == 3:
            sequence, tokens = live.pop(int(rng.integers(0, 3)))
            more = rng.integers(0, config["vocab"], size=2).tolist()
            got = engine.run([(sequence, more, [0, 1])])[0]
            Reference(config, weights, tokens + more).check(got, [len(tokens), len(tokens) + 1], dtype, turn)
            engine.close(sequence)


def test_engine_refuses_what_it_cannot_run(runtime):
    config = MODELS["odd"]
    engine = build(runtime, config, weights_of(config), capacity=16, token_capacity=16, page=8)
    sequence = engine.open()
    for entries, message in (([(sequence, [1] * 17, [])], "capacity is exhausted"), ([(sequence, [61], [])], "outside the vocabulary"),
                             ([(sequence, [1], [1])], "places must lie"), ([(sequence, [], [])], "needs tokens"),
                             ([(5, [1], [])], "not open"), ([(sequence, [1], []), (sequence, [2], [])], "only appear once")):
        with pytest.raises(ValueError, match=message):
            engine.run(entries)
    assert engine.sequences.lengths[sequence] == 0
    with pytest.raises(ValueError, match="unsupported element type"):
        build(runtime, config, weights_of(config), dtype="float16")


# ---- generation ------------------------------------------------------------------------------------------------

def greedy(config, weights, prompt, steps):
    tokens, gaps = list(prompt), []
    for _ in range(steps):
        logits = plain.forward(config, weights, tokens)[-1]
        top = np.sort(logits)[-2:]
        gaps.append((top[1] - top[0]) / logits.std())
        tokens.append(int(np.argmax(logits)))
    return tokens[len(prompt):], min(gaps)


def test_greedy_generation_through_the_engine(runtime):
    """More prompts than places in the batch, unequal lengths: the tokens of the plain restatement."""
    config = MODELS["mixed"]
    weights = weights_of(config, seed=3)
    rng = np.random.default_rng(11)
    prompts = [rng.integers(0, config["vocab"], size=n).tolist() for n in (5, 1, 33, 12, 2)]
    wanted = [greedy(config, weights, prompt, 16) for prompt in prompts]
    assert min(gap for _, gap in wanted) > 1e-4
    engine = build(runtime, config, weights, batch=2, capacity=64, dtype="float32")
    assert engine.generate(prompts, 16) == [tokens for tokens, _ in wanted]
    # a stop token ends its sequence at once and makes room for the next
    stop = wanted[2][0][4]
    cut = lambda tokens: tokens[:tokens.index(stop) + 1] if stop in tokens else tokens
    assert engine.generate(prompts, 16, stop=(stop,)) == [cut(tokens) for tokens, _ in wanted]
    # the lock-step interface, host-driven and chained on the device
    batch = build(runtime, config, weights, batch=2, capacity=64, dtype="float32")
    pair = [prompts[0], [t for t in prompts[0][::-1]]]
    second = greedy(config, weights, pair[1], 16)[0]
    tokens = [batch.prefill(prompt, sequence) for sequence, prompt in enumerate(pair)]
    stream = [tokens]
    for step in range(8):
        stream.append(batch.step(stream[-1], 5 + step))
    assert [t[0] for t in stream] == wanted[0][0][:9] and [t[1] for t in stream] == second[:9]
    chained, elapsed = batch.generate_chained(stream[-1], 13, 7)
    assert chained == wanted[0][0][9:16] and elapsed > 0
    # seeded sampling: the same seed gives the same tokens
    draws = [engine.generate(prompts[:2], 8, temperature=1.0, top_k=20, seed=s) for s in (5, 5, 6)]
    assert draws[0] == draws[1] != draws[2]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(runtime, dtype):
    config = config_of([memory_layer(heads=2, dim=24, vdim=32), parallel_layer()], vocab=90)
    weights = weights_of(config, seed=4)
    tokens = np.random.default_rng(12).integers(0, 90, size=600).tolist()
    engine = build(runtime, config, weights, capacity=640, dtype=dtype)
    sequence = engine.open()
    engine.run([(sequence, tokens[:20], [])])
    got = np.array([engine.run([(sequence, [token], [0])])[0][0] for token in tokens[20:]])
    Reference(config, weights, tokens).check(got, np.arange(20, 600), dtype)


def test_trace_runner(runtime, tmp_path):
    """The program end to end: a checkpoint on disk, steps on standard input, logits in files."""
    import json
    import os
    import subprocess
    import sys

    from llmopt_b200.safetensors_archive import as_bfloat16_bits
    from test_mixers_cpu import write_checkpoint

    config = MODELS["mixed"]
    weights = weights_of(config)
    (tmp_path / "config.json").write_text(json.dumps(config))
    write_checkpoint(tmp_path / "model.safetensors", {name: ("BF16", as_bfloat16_bits(value)) for name, value in weights.items()})
    tokens = np.random.default_rng(13).integers(0, config["vocab"], size=20).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[18:], "want": [1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tokens[:1], "want": [0]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    out.mkdir()
    done = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "24"], input="".join(json.dumps(s) + "\n" for s in steps),
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(4)]
    reference = Reference(config, weights, tokens)
    read = lambda step: np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, config["vocab"])
    reference.check(read(0), [0, 16], "float32")
    reference.check(read(2), [19], "float32")
    reference.check(read(3), [0], "float32")
    assert not (out / "1.f32").exists()


def test_generate_command(runtime, tmp_path, capsys):
    import json

    from llmopt_b200 import generate
    from llmopt_b200.safetensors_archive import as_bfloat16_bits
    from test_mixers_cpu import write_checkpoint

    config = MODELS["mixed"]
    weights = weights_of(config, seed=3)
    (tmp_path / "config.json").write_text(json.dumps(config))
    write_checkpoint(tmp_path / "model.safetensors", {name: ("BF16", as_bfloat16_bits(value)) for name, value in weights.items()})
    generate.main(["--model", str(tmp_path), "--prompt", "3,99,41", "--prompt", "7", "--tokens", "6", "--dtype", "float32"])
    wanted = [greedy(config, weights, prompt, 6)[0] for prompt in ([3, 99, 41], [7])]
    assert capsys.readouterr().out.splitlines() == [",".join(map(str, tokens)) for tokens in wanted]

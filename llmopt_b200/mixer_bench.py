"""Prefill and decode throughput of decoders composed of sequence mixers, and the roofline share of every
kernel of their steps: the recurrent design beside the W4A16 decoder of the same width, depth, heads and vocabulary
and the like kernels of that path, the windowed design with routed experts beside the recurrent one.  Used by
``bench.py --mixers``; random weights.

  python -m llmopt_b200.mixer_bench [--design bizodra|dalorax] [--size 2048|4096|all] [--tokens 2048] [--context 2048]"""

from __future__ import annotations

import argparse
import json
import statistics
import struct
import time
from types import SimpleNamespace

import numpy as np

from . import parameters
from .cuda_native import Batch, Runtime
from .model import (AttentionSpec, DeltaSpec, ExpertsSpec, FeedForwardSpec, MatrixMemorySpec, MixerConfig, MixerLayer,
                    ModelConfig, ParallelSpec, RotarySpec, TokenSideSpec, WindowSpec, YarnSpec, random_mixer_weights,
                    random_weights)


def sized_config(width: int) -> MixerConfig:
    """Eight layers of a real model's proportions: matrix memory with 128 x 256 heads, attention and gated
    delta rule with 128-wide heads, four query heads per key/value head."""
    heads = width // 128
    rotary = RotarySpec(dims=128, base=500000.0, scaling=YarnSpec(factor=4.0, original=8192, fast=32.0, slow=1.0))
    memory = MatrixMemorySpec(heads=heads // 2, dim=128, vdim=256, gate_cap=15.0)
    parallel = ParallelSpec(
        left=AttentionSpec(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, rotary=rotary, bias=True,
                           head_norm=True, sink=True),
        right=DeltaSpec(heads=heads, kv_heads=heads // 2, dim=128, vdim=128, taps=4))
    feed_forward = FeedForwardSpec(width=7 * width // 2)
    layers = tuple(MixerLayer(mixer=parallel if index % 2 else memory, feed_forward=feed_forward) for index in range(8))
    return MixerConfig(name=f"mixers-{width}", width=width, vocabulary=32768, layers=layers, epsilon=1e-5, norm_offset=1.0,
                       token_side=TokenSideSpec(dim=256))


def windowed_config(width: int) -> MixerConfig:
    """The same width, depth, heads, feed-forward width and vocabulary with windowed attention; half of the layers read
    another's keys and values, half have sixteen experts of a quarter of the feed-forward width, two per token."""
    heads = width // 128

    def layer(index):
        attention = AttentionSpec(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, gate=True,
                                  weights32=True, window=WindowSpec(size=1024, keep_first=4),
                                  kv_from=index // 4 * 4 + 1 if index % 4 >= 2 else None)
        routed = ExpertsSpec(experts=16, top=2, width=7 * width // 8)
        return MixerLayer(mixer=attention, feed_forward=routed if index % 2 else FeedForwardSpec(
            width=7 * width // 2, activation="silu", gated=True))

    return MixerConfig(name=f"windows-{width}", width=width, vocabulary=32768, layers=tuple(layer(index) for index in range(8)),
                       epsilon=1e-5, norm="tanh", sinusoid=True, tied_head=True)


def like_config(config: MixerConfig) -> ModelConfig:
    """The W4A16 decoder of the same size."""
    heads = config.width // 128
    return ModelConfig(f"w4a16-{config.width}", config.width, ("attention",) * len(config.layers), heads, heads // 4, 128,
                       config.layers[0].feed_forward.width, config.vocabulary)


# ---- algorithmic work of a dispatch ------------------------------------------------------------------------

def experts_in_use(item) -> int:
    """Experts that some row of an expert kernel's step chose, from its device-side route or plan."""
    words = item.buffers[2].to_numpy(np.uint32)
    if "expert_step" in item.name:
        return int(words[0])
    return len(set(words[4:4 + 4 * int(words[0])].reshape(-1, 4)[:, 0].tolist()))


def work_of(item, past: int, itemsize: int):
    """(label, bytes, flops) of a recorded dispatch; every operand once."""
    stem = item.name.removeprefix("llmopt_").removesuffix("_bf16").removesuffix("_f32")
    u = struct.unpack(f"<{len(item.parameters) // 4}I", item.parameters)
    e = itemsize
    if stem == "dense_linear":
        m, n, k, split = u[:4]
        if u[5] == parameters.DENSE_EPILOGUES["silu_pair"]:
            return f"dense_linear (pairs) n{n} k{k}", n * k * e + m * k * e + m * n // 2 * e, 2 * m * n * k
        return f"dense_linear n{n} k{k}", n * k * e + m * k * e + m * split * e + m * (n - split) * 4, 2 * m * n * k
    if stem == "dense_cached":
        m, n, k = u[:3]
        return f"dense_cached n{n} k{k}", (n * k + m * k + m * n) * e, 2 * m * n * k
    if stem == "dense_residual":
        m, n, k = u[:3]
        return f"dense_residual n{n} k{k}", (n * k + m * k + m * n) * e + m * n * 8, 2 * m * n * k
    if stem in ("expert_step", "expert_step_residual"):
        rows, n, k, experts, top = u
        used = experts_in_use(item)
        edges = rows * k + used * rows * n // 2 if stem == "expert_step" else used * rows * k + rows * n
        return f"{stem} n{n} k{k}", (used * n * k + edges) * e + (rows * n * 8 if "residual" in stem else 0), 2 * rows * top * n * k
    if stem == "expert_rows":
        pairs, n, k, experts, paired = u
        return (f"expert_rows n{n} k{k}", (experts_in_use(item) * n * k + pairs * k) * e + pairs * n * (e // 2 if paired else 4),
                2 * pairs * n * k)
    if stem in ("route_step", "route_rows", "route_plan"):
        rows, experts, top = u
        return stem, rows * (experts * 4 if stem != "route_plan" else top * 8) + rows * top * (8 if stem != "route_plan" else 12), 0
    if stem == "expert_combine":
        rows, width, top = u
        return stem, rows * width * (4 * top + 8 + e), 0
    if stem == "embedding_sinusoid":
        return stem, u[0] * u[3] * (2 * e + 4), 0
    if stem == "gather_rows":
        return stem, u[0] * u[2] * 2 * e, 0
    if stem == "embedding_residual":
        return stem, u[0] * u[2] * (2 * e + 4), 0
    if stem == "residual_norm":
        rows, width, _, _, pair = u
        return stem + (" (two branches)" if pair else ""), rows * width * (4 + 4 + (4 if pair else 0) + 4 + e), 0
    if stem == "gather_norm":
        return stem, u[0] * u[2] * (4 + e), 0
    if stem == "row_attention_prepare":
        sequences, tokens, heads, kv_heads, dim, vdim = u[:6]
        return stem, sequences * tokens * 2 * e * (heads * dim + kv_heads * (dim + vdim)), 0
    if stem == "row_attention":
        sequences, tokens, heads, kv_heads, dim, vdim = u[:6]
        window, keep_first, gated = u[16], u[17], u[20] > 0
        keys, pairs = past + tokens, tokens * past + tokens * (tokens + 1) // 2
        if window:
            seen = [min(past + t + 1, window + min(keep_first, max(0, past + t + 1 - window))) for t in range(tokens)]
            pairs, keys = sum(seen), min(keys, window + tokens - 1 + keep_first)
        if gated:
            stem += " (windowed, gated)"
        return (stem, sequences * (keys * kv_heads * (dim + vdim) * e + tokens * heads * (dim + vdim + (vdim if gated else 0)) * e),
                2 * sequences * heads * pairs * (dim + vdim))
    if stem == "head_norm_gate":
        return stem, u[0] * u[1] * u[2] * (4 + 2 * e), 0
    if stem in ("delta_prepare", "conv_state"):
        sequences, tokens, heads, kv_heads, dim, vdim, taps = u[:7]
        channels = 2 * kv_heads * dim + heads * vdim
        if stem == "conv_state":
            return stem, sequences * channels * (taps - 1) * 2 * e, 0
        return stem, sequences * tokens * (channels * (e + 4) + heads * 16), 0
    if stem in ("delta_scan", "memory_scan"):
        sequences, tokens, heads, kv_heads, dim, vdim = u[:6]
        source = 4 if stem == "delta_scan" else e
        vectors = (2 * kv_heads * dim + heads * vdim) * source + heads * (vdim * 4 + 8)
        return stem, sequences * (tokens * vectors + heads * dim * vdim * 8), 0
    if stem in ("delta_step", "memory_step"):
        sequences, heads, kv_heads, dim, vdim = u[0], u[2], u[3], u[4], u[5]  # u[1]: one token
        return stem, sequences * (heads * dim * vdim * 8 + (2 * kv_heads * dim + 3 * heads * vdim) * e), 0
    if stem == "argmax":
        return stem, u[0] * u[1] * 4, 0
    return stem, 0, 0


def time_items(runtime, items, past: int, itemsize: int, peaks: dict) -> dict:
    """Per kernel: all its launches of the step back to back (every layer's own operands)."""
    groups = {}
    for item in items:
        groups.setdefault(work_of(item, past, itemsize)[0], []).append(item)
    table = {}
    for label, group in groups.items():
        if label.startswith(("route", "expert")):
            runtime.time_dispatches(items, warmup=0, iterations=1)  # routes of a whole step, not of what was timed before
        launches = len(group)
        ms = runtime.time_dispatches(group * max(1, min(16, 64 // launches)), warmup=2, iterations=5)
        _, nbytes, flops = work_of(group[0], past, itemsize)
        floor = max(nbytes / peaks["hbm_gbs"] / 1e6, flops / peaks["bf16_tflops"] / 1e9)
        table[label] = {"launches": launches, "us": round(ms * 1e3, 2), "floor_us": round(floor * 1e3, 2),
                        "frac": round(floor / ms, 3) if ms else None, "share_us": round(ms * 1e3 * launches, 1)}
        if label.startswith("expert") and "combine" not in label:
            table[label]["experts_in_use"] = experts_in_use(group[0])
    return table


# ---- whole steps ---------------------------------------------------------------------------------------------

def decode_rate(engine, batch: int, context: int, steps: int = 32) -> dict:
    if hasattr(engine, "rewind"):
        engine.rewind(context)
    first = [1 + index for index in range(batch)]
    engine.generate_chained(first, context, 8)
    times = []
    for _ in range(5):
        if hasattr(engine, "rewind"):
            engine.rewind(context)
        _, elapsed = engine.generate_chained(first, context, steps)
        times.append(elapsed / steps)
    ms = statistics.median(times)
    return {"batch": batch, "context": context, "ms_per_step": round(ms, 4), "tokens_per_s": round(batch * 1e3 / ms, 1)}


def prefill_rate(engine, tokens: int) -> dict:
    prompt = np.random.default_rng(0).integers(0, engine.config.vocabulary, size=tokens).tolist()
    engine.prefill(prompt)
    times = []
    for _ in range(5):
        engine.runtime.synchronize()
        started = time.perf_counter()
        engine.prefill(prompt)
        times.append(time.perf_counter() - started)
    seconds = statistics.median(times)
    return {"tokens": tokens, "ms": round(seconds * 1e3, 3), "tokens_per_s": round(tokens / seconds, 1)}


def measure_mixers(runtime, peaks: dict, config: MixerConfig, tokens: int, context: int, batches=(1, 8, 32)) -> dict:
    from .mixer_engine import MixerEngine

    weights = random_mixer_weights(config, seed=0, fast=True)
    result = {"model": config.name, "width": config.width, "layers": len(config.layers), "decode": [], "kernels": {}}
    for batch in batches:
        engine = MixerEngine(runtime, config, weights, batch=batch, capacity=context + 64 + (tokens if batch == 1 else 0),
                             prompt_rows=tokens if batch == 1 else batch)
        result["decode"].append(decode_rate(engine, batch, context))
        plan = engine._decode_plan(batch)[0]
        engine.rewind(context)
        plan.write(list(range(1, batch + 1)), [context] * batch, [engine._row(index) for index in range(batch)])
        items = [item for item in plan.items if item.name != "llmopt_advance_tokens"]
        result["kernels"][f"decode, {batch} sequences, {context} tokens behind"] = time_items(
            runtime, items, context, engine.itemsize, peaks)
        result["decode"][-1]["kernels_per_step"] = engine._decode_plan(batch)[1].kernel_count()
        if batch == 1:
            result["prefill"] = prefill_rate(engine, tokens)
            plan = engine._prompt_plan(tokens)[0]
            plan.write(np.random.default_rng(0).integers(0, config.vocabulary, size=tokens), [0], [engine._row(0)])
            result["kernels"][f"prompt of {tokens} tokens"] = time_items(runtime, plan.items, 0, engine.itemsize, peaks)
    return result


def measure_like(runtime, peaks: dict, config: MixerConfig, tokens: int, context: int, batches=(1, 8, 32)) -> dict:
    from .decode_engine import DecodeEngine

    like = like_config(config)
    weights = random_weights(like, seed=0, fast=True)
    result = {"model": like.name, "width": like.hidden, "layers": len(like.layers), "decode": []}
    for batch in batches:
        engine = DecodeEngine(runtime, like, weights, batch=batch, capacity=context + 64 + tokens)
        engine.fill_cache_random(context)
        engine.build(context)
        result["decode"].append(decode_rate(engine, batch, context))
        if batch == 1:
            result["prefill"] = prefill_rate(engine, tokens)
    return result


def like_kernels(runtime, peaks: dict, config: MixerConfig, tokens: int, context: int) -> dict:
    """The like kernels of the W4A16 path at the same sizes: share of the roofline of each."""
    from . import dispatch, kernel_bench
    from .cuda_native import Buffer, DispatchItem

    width, heads = config.width, config.width // 128
    table = {}

    def note(label, ms, nbytes, flops=0.0):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e6, flops / peaks["bf16_tflops"] / 1e9)
        table[label] = {"us": round(ms * 1e3, 2), "floor_us": round(floor * 1e3, 2), "frac": round(floor / ms, 3)}

    def probe(label, op, copies, flops=0.0, **options):
        args = SimpleNamespace(op=op, m=1, k=width, n=7 * width // 2, heads=heads, kv_heads=heads // 4, dim=128, group=64, layers=2,
                               past=context)
        args.__dict__.update(options)
        keep, items = [], []
        for _ in range(copies):
            item, nbytes, context_ = kernel_bench.build_item(runtime, args)
            keep.append(context_)
            items.append(item)
        note(label, runtime.time_dispatches(items, warmup=2, iterations=5), nbytes, flops)

    for m in (1, 8, 32):
        probe(f"w4a16 linear n{3 * width} k{width}, {m} rows", "linear", 24, m=m, n=3 * width)
        probe(f"w4a16 linear n{width} k{width}, {m} rows", "linear", 64, m=m, n=width)
        probe(f"paged attention q8, {m} sequences", "attention", 8, m=m)
    probe(f"w4a16 linear n{7 * width // 2} k{width}, {tokens} rows", "linear", 8, m=tokens, flops=2.0 * tokens * width * 7 * width // 2)
    probe(f"w4a16 linear n{width} k{width}, {tokens} rows", "linear", 8, m=tokens, n=width, flops=2.0 * tokens * width * width)
    probe(f"dense attention, {tokens} tokens", "dense_attention", 2, m=tokens, flops=2.0 * tokens * tokens * 128 * heads)
    rng = np.random.default_rng(0)
    half = lambda *shape: dispatch.Tensor(Buffer.of_array(runtime, (rng.standard_normal(shape) * 0.1).astype(np.float16)), shape)
    commands = Batch(runtime)
    recurrent = dispatch.Context(runtime, batch=commands)
    for count in (tokens, 1):
        q, k, v, beta, out = (half(1, count, heads, 128), half(1, count, heads, 128), half(1, count, heads, 128),
                              half(1, count, heads), half(1, count, heads, 128))
        gate = dispatch.Tensor(Buffer.of_array(runtime, -np.ones((1, count, heads), np.float32)), (1, count, heads), "float32")
        dispatch.dispatch_gated_delta(recurrent, query=q, key=k, value=v, gate=gate, beta=beta, output=out)
        note(f"gated delta scan (from a zero state), {count} tokens",
             runtime.time_dispatches([commands.pending.pop()] * 4, warmup=1, iterations=3), count * heads * (128 * 8 + 6))
        rows = half(count, width)
        item = DispatchItem("llmopt_rms_norm_f16_simd", [rows.buffer, half(width).buffer, half(count, width).buffer],
                            parameters.rms_norm(rows=count, width=width, epsilon=1e-5),
                            (dispatch.simd_rows_grid(count), 1, 1), (256, 1, 1))
        note(f"rms norm, {count} rows", runtime.time_dispatches([item] * 32, warmup=2, iterations=5), count * width * 4)
        q_in, k_in = half(count, heads * 128), half(count, heads // 4 * 128)
        rotary = DispatchItem("llmopt_rotary_qk_f16_simd_h64",
                              [q_in.buffer, k_in.buffer, half(count, 128).buffer, half(count, 128).buffer,
                               half(count, heads * 128).buffer, half(count, heads // 4 * 128).buffer],
                              parameters.rotary_qk(batches=1, tokens=count, q_heads=heads, k_heads=heads // 4, width=128,
                                                   half_dimension=64, trig_batches=1),
                              (dispatch.simd_rows_grid(count * (heads + heads // 4)), 1, 1), (256, 1, 1))
        note(f"rotary q k, {count} rows", runtime.time_dispatches([rotary] * 16, warmup=2, iterations=5),
             count * (heads + heads // 4) * 128 * 4)
        conv = DispatchItem("llmopt_short_conv_silu_tm_f16", [rows.buffer, half(width, 4).buffer, half(count, width).buffer],
                            parameters.short_conv_silu_tm(batches=1, tokens=count, channels=width, kernel_width=4, stride=1,
                                                          padding=3, dilation=1, output_start=0), (1, 1, 1), (256, 1, 1))
        note(f"short conv + silu, {count} rows", runtime.time_dispatches([conv] * 16, warmup=2, iterations=5), count * width * 4)
    commands.abort()
    return table


def measure(runtime, peaks: dict, widths=(2048, 4096), tokens: int = 2048, context: int = 2048, like: bool = True,
            design: str = "bizodra") -> list:
    results = []
    for width in widths:
        config = sized_config(width)
        if design == "dalorax":
            entry = {"windows": measure_mixers(runtime, peaks, windowed_config(width), tokens, context)}
            if like:
                entry["mixers"] = measure_mixers(runtime, peaks, config, tokens, context)
        else:
            entry = {"mixers": measure_mixers(runtime, peaks, config, tokens, context)}
            if like:
                entry["w4a16"] = measure_like(runtime, peaks, config, tokens, context)
                entry["w4a16_kernels"] = like_kernels(runtime, peaks, config, tokens, context)
        results.append(entry)
    return results


def main() -> None:
    parser = argparse.ArgumentParser()
    parser.add_argument("--design", default="bizodra", choices=["bizodra", "dalorax"])
    parser.add_argument("--size", default="all", choices=["2048", "4096", "all"])
    parser.add_argument("--tokens", type=int, default=2048)
    parser.add_argument("--context", type=int, default=2048)
    parser.add_argument("--no-like", action="store_true", help="only the design itself")
    args = parser.parse_args()
    peaks = {"hbm_gbs": 6531.6, "bf16_tflops": 1657.8}
    widths = (2048, 4096) if args.size == "all" else (int(args.size),)
    for entry in measure(Runtime(), peaks, widths, args.tokens, args.context, not args.no_like, args.design):
        print(json.dumps(entry, indent=1))


if __name__ == "__main__":
    main()

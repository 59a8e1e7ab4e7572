"""Record builders of the sequence mixers: what a layer of a ``model.MixerConfig`` dispatches.

A mixer declares the projections of its input that it reads (the engine computes all of a layer's in one
product), owns its weights and its per-sequence state on the device, and records the kernels from the
projected rows to the product that ends the sublayer (``residual``).  ``LayerMixer`` runs one, or two of them
side by side.

The engine (``mixer_engine.MixerEngine``) hands a ``Step`` to the builders: the shape of the step and the
device buffers every kernel of it reads."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Tuple

import numpy as np

from . import parameters
from .cuda_native import Buffer
from .kv_cache import MATRIX_STATE_SLICE, matrix_state_elements
from .model import AttentionSpec, DeltaSpec, MatrixMemorySpec, ParallelSpec


@dataclass
class Step:
    """``sequences`` sequences with ``tokens`` rows each (row = sequence * tokens + token)."""

    engine: object
    sequences: int
    tokens: int
    ids: Buffer            # i64 [rows]
    past: Buffer           # u32 [sequences]: tokens behind the step
    sequence_rows: Buffer  # u32 [sequences]: row of the slot table and of the state pools
    run: object            # run(name, buffers, parameters) records a dispatch
    stream: object = None  # residual stream of the step (``residual``), once its layers are recorded

    @property
    def rows(self) -> int:
        return self.sequences * self.tokens

    def element(self, stem: str) -> str:
        return f"llmopt_{stem}_{self.engine.suffix}"


class Projection:
    """All projections of a layer's mixer input as one weight matrix: parts read in the model's element
    type first, then keys and values that go straight into the cache, then the parts that feed fp32 arithmetic."""

    ORDER = ("element", "cache", "fp32")

    def __init__(self):
        self.parts: List[Tuple[str, np.ndarray, object, str]] = []
        self.region = None  # cache region of the "cache" parts

    def add(self, key: str, weight: np.ndarray, bias=None, fp32: bool = False, cache: bool = False) -> None:
        self.parts.append((key, weight, bias, "cache" if cache else "fp32" if fp32 else "element"))

    def upload(self, engine) -> None:
        ordered = sorted(self.parts, key=lambda part: self.ORDER.index(part[3]))
        self.columns: Dict[str, int] = {}
        rows = {kind: [weight.shape[0] for _, weight, _, k in ordered if k == kind] for kind in self.ORDER}
        self.split, self.scalars, self.cached = sum(rows["element"]), sum(rows["fp32"]), rows["cache"]
        self.total = self.split + sum(self.cached) + self.scalars
        start = dict(zip(self.ORDER, (0, self.split, self.split + sum(self.cached))))
        total = 0
        for key, weight, _, kind in ordered:
            self.columns[key] = total - start[kind]
            total += weight.shape[0]
        self.weight = engine.upload_matrix(np.concatenate([np.ascontiguousarray(w) for _, w, _, _ in ordered]))
        self.bias = None
        if any(bias is not None for _, _, bias, _ in ordered):
            from .safetensors_archive import as_float32

            self.bias = engine.upload_vector(np.concatenate(
                [np.zeros(weight.shape[0], np.float32) if bias is None else as_float32(bias) for _, weight, bias, _ in ordered]))
        self.parts = []

    def record(self, step: Step, x: Buffer):
        """(rows in the element type, fp32 rows)."""
        engine = step.engine
        projected, scalars = engine.work("projected", self.split), engine.work32("scalars", max(self.scalars, 1))
        if self.cached:
            keys, values = self.cached
            step.run(step.element("dense_cached"),
                     [x, self.weight, self.bias or self.weight, projected, scalars, engine.token_pool, engine.slot_table, step.past,
                      step.sequence_rows],
                     parameters.dense_cached(m=step.rows, n=self.total, k=engine.config.width, split=self.split, tokens=step.tokens,
                                             key_columns=keys, value_columns=values, has_bias=self.bias is not None,
                                             **engine.cache_rows(self.region)))
        else:
            engine.record_linear(step, x, self.weight, projected, m=step.rows, n=self.total, k=engine.config.width,
                                 split=self.split, out32=scalars, bias=self.bias)
        return projected, scalars


def fused_step(step: Step, spec) -> bool:
    """Whether the one-launch form of a recurrent mixer takes this step: one token per sequence, a head's
    value columns fit the thread blocks of one cluster, and there are few enough of those blocks for the
    step to be a matter of launches rather than of state traffic (which the scan streams better)."""
    slices = (spec.vdim + MATRIX_STATE_SLICE - 1) // MATRIX_STATE_SLICE
    return step.tokens == 1 and slices <= 8 and step.sequences * spec.heads * slices <= 2048


class AttentionMixer:
    """Causal attention over the unquantised row cache.  Where queries and keys are used as they are projected
    (no head norm, no rotation), the projection writes keys and values into the cache and the scores read the queries
    from its rows; otherwise a kernel between the two prepares them."""

    def __init__(self, engine, spec: AttentionSpec, weights, prefix: str, projection: Projection, layer: int, branch: int):
        self.spec, self.projection, self.prefix, self.branch = spec, projection, prefix, branch
        self.region = engine.attention_region(layer, spec)
        self.own_keys = spec.kv_from is None
        direct = self.own_keys and not spec.prepared and projection.region is None
        bias = (lambda name: weights[f"{prefix}.{name}.b"]) if spec.bias else (lambda name: None)
        projection.add(f"{prefix}.q", weights[f"{prefix}.q"], bias("q"))
        if spec.gate:
            projection.add(f"{prefix}.g", weights[f"{prefix}.g"])
        if self.own_keys:
            for name in "kv":
                projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"], bias(name), cache=direct)
        if direct:
            projection.region = self.region
        self.prepares = not direct and (self.own_keys or spec.prepared)
        self.out = engine.upload_matrix(weights[f"{prefix}.o"])
        self.out_bias = engine.upload_vector(bias("o")) if spec.bias else None
        self.head_norms = [engine.upload_vector(weights[f"{prefix}.{name}.norm"]) for name in ("qk" if self.own_keys else "qq")
                           ] if spec.head_norm else None
        self.trig = engine.rotary_table(spec.rotary) if spec.rotary else None

    def record(self, step: Step, projected: Buffer, scalars: Buffer) -> None:
        engine, spec, columns = step.engine, self.spec, self.projection.columns
        attended = engine.work("mixed", spec.heads * spec.vdim)
        shape = dict(sequences=step.sequences, tokens=step.tokens, heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim,
                     vdim=spec.vdim)
        cache = engine.cache_rows(self.region)
        stride, column = self.projection.split, lambda name: columns[f"{self.prefix}.{name}"]
        query, queries = projected, dict(query_stride=stride, query_column=column("q"))
        if self.prepares:
            query, queries = engine.work("query", spec.heads * spec.dim), {}
            trig = self.trig or projected
            q_norm, k_norm = self.head_norms or (trig, trig)
            step.run(step.element("row_attention_prepare"),
                     [projected, q_norm, k_norm, trig, query, engine.token_pool, engine.slot_table, step.past, step.sequence_rows],
                     parameters.row_attention_prepare(
                         **shape, stride=stride, q_column=column("q"), k_column=column("k") if self.own_keys else 0,
                         v_column=column("v") if self.own_keys else 0, rotary_dims=spec.rotary.dims if spec.rotary else 0,
                         trig_rows=engine.capacity, **cache, head_norm=spec.head_norm, epsilon=engine.config.epsilon,
                         own_keys=self.own_keys))
        gate = dict(gate_stride=stride, gate_column=column("g")) if spec.gate else {}
        window = dict(window=spec.window.size, keep_first=spec.window.keep_first) if spec.window else {}
        splits, scratch = engine.attention_splits(step, spec)
        step.run(step.element("row_attention"),
                 [query, engine.token_pool, engine.slot_table, step.past, step.sequence_rows, attended, scratch, projected],
                 parameters.row_attention(**shape, **cache, sink=spec.sink, splits=splits, scale=spec.scale,
                                          softcap=spec.softcap or 0.0, weights32=spec.weights32, **queries, **gate, **window))
        step.stream.product(attended, self.out, k=spec.heads * spec.vdim, bias=self.out_bias, branch=self.branch)


class DeltaMixer:
    """Gated delta rule over short-convolved, unit-length q and k."""

    def __init__(self, engine, spec: DeltaSpec, weights, prefix: str, projection: Projection, layer: int, branch: int):
        from .safetensors_archive import as_float32

        self.spec, self.projection, self.prefix, self.branch = spec, projection, prefix, branch
        for name in "qkvg":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"])
        for name in "ba":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"], fp32=True)
        self.conv = engine.upload_vector(np.concatenate([as_float32(weights[f"{prefix}.{name}.conv"]) for name in "qkv"]))
        self.a_log, self.dt_bias, self.norm, = (engine.upload_vector(weights[f"{prefix}.{name}"])
                                                for name in ("A_log", "dt_bias", "norm"))
        self.out = engine.upload_matrix(weights[f"{prefix}.o"])
        self.channels = 2 * spec.kv_heads * spec.dim + spec.heads * spec.vdim
        self.state_stride = matrix_state_elements(spec.heads, spec.dim, spec.vdim, normalized=False)
        rows = engine.sequences.rows
        self.state = engine.empty_bytes(rows * self.state_stride * 4)
        self.conv_state = engine.empty_bytes(rows * self.channels * spec.taps * engine.itemsize)

    def record(self, step: Step, projected: Buffer, scalars: Buffer) -> None:
        engine, spec, columns = step.engine, self.spec, self.projection.columns
        qk, vs = spec.kv_heads * spec.dim, spec.heads * spec.vdim
        q, k, v = engine.work32("delta_q", qk), engine.work32("delta_k", qk), engine.work32("delta_v", vs)
        decay, beta = engine.work32("delta_decay", spec.heads), engine.work32("delta_beta", spec.heads)
        read_out, mixed = engine.work32("read_out", vs), engine.work("mixed", vs)
        shape = dict(sequences=step.sequences, tokens=step.tokens, heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim,
                     vdim=spec.vdim)
        rows = engine.sequences.rows
        if fused_step(step, spec):
            step.run(step.element("delta_step"),
                     [projected, scalars, self.conv, self.conv_state, self.a_log, self.dt_bias, self.norm, self.state, step.past,
                      step.sequence_rows, mixed],
                     parameters.state_step(
                         sequences=step.sequences, heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim, vdim=spec.vdim,
                         taps=spec.taps, stride=self.projection.split, q_column=columns[f"{self.prefix}.q"],
                         k_column=columns[f"{self.prefix}.k"], v_column=columns[f"{self.prefix}.v"],
                         gate_column=columns[f"{self.prefix}.g"], scalar_stride=self.projection.scalars,
                         first_column=columns[f"{self.prefix}.b"], second_column=columns[f"{self.prefix}.a"], state_rows=rows,
                         state_stride=self.state_stride, gate_cap=0.0, epsilon=engine.config.epsilon))
            step.stream.product(mixed, self.out, k=vs, branch=self.branch)
            return
        prepare = parameters.delta_prepare(
            **shape, taps=spec.taps, stride=self.projection.split, q_column=columns[f"{self.prefix}.q"],
            k_column=columns[f"{self.prefix}.k"], v_column=columns[f"{self.prefix}.v"],
            scalar_stride=self.projection.scalars, beta_column=columns[f"{self.prefix}.b"],
            decay_column=columns[f"{self.prefix}.a"], state_rows=rows)
        step.run(step.element("delta_prepare"),
                 [projected, scalars, self.conv, self.conv_state, step.past, step.sequence_rows, self.a_log, self.dt_bias,
                  q, k, v, decay, beta], prepare)
        step.run(step.element("conv_state"), [projected, self.conv_state, step.past, step.sequence_rows], prepare)
        step.run("llmopt_delta_scan_f32", [q, k, v, decay, beta, self.state, step.past, step.sequence_rows, read_out],
                 parameters.state_scan(**shape, q_stride=qk, q_column=0, k_stride=qk, k_column=0, v_stride=vs, v_column=0,
                                       scalar_stride=spec.heads, first_column=0, second_column=0, state_rows=rows,
                                       state_stride=self.state_stride))
        step.run(step.element("head_norm_gate"), [read_out, projected, self.norm, mixed],
                 parameters.head_norm_gate(rows=step.rows, heads=spec.heads, dim=spec.vdim,
                                           gate_stride=self.projection.split, gate_column=columns[f"{self.prefix}.g"],
                                           weight_per_head=False, gate_sigmoid=False, epsilon=engine.config.epsilon))
        step.stream.product(mixed, self.out, k=vs, branch=self.branch)


class MatrixMemoryMixer:
    """Matrix memory with stabilised exponential input and forget gates."""

    def __init__(self, engine, spec: MatrixMemorySpec, weights, prefix: str, projection: Projection, layer: int, branch: int):
        self.spec, self.projection, self.prefix, self.branch = spec, projection, prefix, branch
        for name in "qkvg":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"])
        for name in "if":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"], weights[f"{prefix}.{name}.b"], fp32=True)
        self.norm = engine.upload_vector(weights[f"{prefix}.norm"])
        self.out = engine.upload_matrix(weights[f"{prefix}.o"])
        self.state_stride = matrix_state_elements(spec.heads, spec.dim, spec.vdim, normalized=True)
        self.state = engine.empty_bytes(engine.sequences.rows * self.state_stride * 4)

    def record(self, step: Step, projected: Buffer, scalars: Buffer) -> None:
        engine, spec, columns = step.engine, self.spec, self.projection.columns
        vs, stride = spec.heads * spec.vdim, self.projection.split
        read_out, mixed = engine.work32("read_out", vs), engine.work("mixed", vs)
        if fused_step(step, spec):
            step.run(step.element("memory_step"),
                     [projected, scalars, self.norm, self.state, step.past, step.sequence_rows, mixed],
                     parameters.state_step(
                         sequences=step.sequences, heads=spec.heads, kv_heads=spec.heads, dim=spec.dim, vdim=spec.vdim, taps=0,
                         stride=stride, q_column=columns[f"{self.prefix}.q"], k_column=columns[f"{self.prefix}.k"],
                         v_column=columns[f"{self.prefix}.v"], gate_column=columns[f"{self.prefix}.g"],
                         scalar_stride=self.projection.scalars, first_column=columns[f"{self.prefix}.i"],
                         second_column=columns[f"{self.prefix}.f"], state_rows=engine.sequences.rows,
                         state_stride=self.state_stride, gate_cap=spec.gate_cap, epsilon=engine.config.epsilon))
            step.stream.product(mixed, self.out, k=vs, branch=self.branch)
            return
        step.run(step.element("memory_scan"),
                 [projected, projected, projected, scalars, scalars, self.state, step.past, step.sequence_rows, read_out],
                 parameters.state_scan(
                     sequences=step.sequences, tokens=step.tokens, heads=spec.heads, kv_heads=spec.heads, dim=spec.dim,
                     vdim=spec.vdim, q_stride=stride, q_column=columns[f"{self.prefix}.q"], k_stride=stride,
                     k_column=columns[f"{self.prefix}.k"], v_stride=stride, v_column=columns[f"{self.prefix}.v"],
                     scalar_stride=self.projection.scalars, first_column=columns[f"{self.prefix}.i"],
                     second_column=columns[f"{self.prefix}.f"], state_rows=engine.sequences.rows,
                     state_stride=self.state_stride, gate_cap=spec.gate_cap))
        step.run(step.element("head_norm_gate"), [read_out, projected, self.norm, mixed],
                 parameters.head_norm_gate(rows=step.rows, heads=spec.heads, dim=spec.vdim, gate_stride=stride,
                                           gate_column=columns[f"{self.prefix}.g"], weight_per_head=True,
                                           gate_sigmoid=True, epsilon=engine.config.epsilon))
        step.stream.product(mixed, self.out, k=vs, branch=self.branch)


SINGLE_MIXERS = {AttentionSpec: AttentionMixer, DeltaSpec: DeltaMixer, MatrixMemorySpec: MatrixMemoryMixer}


class LayerMixer:
    """A layer's mixer: one, or two side by side whose normed outputs the residual norm averages."""

    def __init__(self, engine, spec, weights, prefix: str, layer: int):
        self.projection = Projection()
        self.branch_norms = None
        if isinstance(spec, ParallelSpec):
            self.branches = [SINGLE_MIXERS[type(one)](engine, one, weights, f"{prefix}.{side}", self.projection, layer, branch)
                             for branch, (side, one) in enumerate((("left", spec.left), ("right", spec.right)))]
            self.branch_norms = [engine.upload_vector(weights[f"{prefix}.{side}.out"]) for side in ("left", "right")]
        else:
            self.branches = [SINGLE_MIXERS[type(spec)](engine, spec, weights, prefix, self.projection, layer, 0)]
        self.projection.upload(engine)

    def record(self, step: Step) -> None:
        projected, scalars = self.projection.record(step, step.stream.x)
        for branch in self.branches:
            branch.record(step, projected, scalars)


def attention_specs(config) -> list:
    """(layer, attention mixer) of every cache region of a model: one per mixer with keys and values of its own."""
    return [(index, spec) for index, layer in enumerate(config.layers) for spec in layer.mixers
            if isinstance(spec, AttentionSpec) and spec.kv_from is None]

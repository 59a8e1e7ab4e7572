"""Record builders of the sequence mixers: what a layer of a ``model.MixerConfig`` dispatches.

A mixer declares the projections of its input that it reads (the engine computes all of a layer's in one
product), owns its weights and its per-sequence state on the device, and records the kernels from the
projected rows to its output, one fp32 row of the model's width per token.  ``ParallelMixer`` runs
two of them side by side.

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

    @property
    def rows(self) -> int:
        return self.sequences * self.tokens

    def element(self, stem: str) -> str:
        return f"llmopt_{stem}_{self.engine.suffix}"


class Projection:
    """All projections of a layer's mixer input as one weight matrix: parts read in the model's element
    type first, then the parts that feed fp32 arithmetic."""

    def __init__(self):
        self.parts: List[Tuple[str, np.ndarray, object, bool]] = []

    def add(self, key: str, weight: np.ndarray, bias=None, fp32: bool = False) -> None:
        self.parts.append((key, weight, bias, fp32))

    def upload(self, engine) -> None:
        ordered = [p for p in self.parts if not p[3]] + [p for p in self.parts if p[3]]
        self.columns: Dict[str, int] = {}
        self.split = sum(weight.shape[0] for _, weight, _, fp32 in ordered if not fp32)
        total = 0
        for key, weight, _, fp32 in ordered:
            self.columns[key] = total - (self.split if fp32 else 0)
            total += weight.shape[0]
        self.total, self.scalars = total, total - self.split
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
    """Causal attention over the unquantised row cache."""

    def __init__(self, engine, spec: AttentionSpec, weights, prefix: str, projection: Projection):
        self.spec, self.projection, self.prefix = spec, projection, prefix
        self.region = engine.next_attention_region()
        bias = (lambda name: weights[f"{prefix}.{name}.b"]) if spec.bias else (lambda name: None)
        for name in "qkv":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"], bias(name))
        self.out = engine.upload_matrix(weights[f"{prefix}.o"])
        self.out_bias = engine.upload_vector(bias("o")) if spec.bias else None
        self.head_norms = [engine.upload_vector(weights[f"{prefix}.{name}.norm"]) for name in "qk"] if spec.head_norm else None
        self.trig = engine.rotary_table(spec.rotary)

    def record(self, step: Step, projected: Buffer, scalars: Buffer, y: Buffer) -> None:
        engine, spec, columns = step.engine, self.spec, self.projection.columns
        query = engine.work("query", spec.heads * spec.dim)
        attended = engine.work("mixed", spec.heads * spec.vdim)
        shape = dict(sequences=step.sequences, tokens=step.tokens, heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim,
                     vdim=spec.vdim)
        cache = dict(token_stride=engine.layout.token_elements, key_offset=self.region.key_offset,
                     value_offset=self.region.value_offset, table_stride=engine.sequences.stride,
                     table_rows=engine.sequences.rows, pool_rows=engine.token_capacity)
        q_norm, k_norm = self.head_norms or (self.trig, self.trig)
        step.run(step.element("row_attention_prepare"),
                 [projected, q_norm, k_norm, self.trig, query, engine.token_pool, engine.slot_table, step.past,
                  step.sequence_rows],
                 parameters.row_attention_prepare(
                     **shape, stride=self.projection.split, q_column=columns[f"{self.prefix}.q"],
                     k_column=columns[f"{self.prefix}.k"], v_column=columns[f"{self.prefix}.v"],
                     rotary_dims=spec.rotary.dims, trig_rows=engine.capacity, **cache, head_norm=spec.head_norm,
                     epsilon=engine.config.epsilon))
        splits, scratch = engine.attention_splits(step, spec)
        step.run(step.element("row_attention"),
                 [query, engine.token_pool, engine.slot_table, step.past, step.sequence_rows, attended, scratch],
                 parameters.row_attention(**shape, **cache, sink=spec.sink, splits=splits, scale=spec.scale))
        engine.record_linear(step, attended, self.out, None, m=step.rows, n=engine.config.width,
                             k=spec.heads * spec.vdim, split=0, out32=y, bias=self.out_bias)


class DeltaMixer:
    """Gated delta rule over short-convolved, unit-length q and k."""

    def __init__(self, engine, spec: DeltaSpec, weights, prefix: str, projection: Projection):
        from .safetensors_archive import as_float32

        self.spec, self.projection, self.prefix = spec, projection, prefix
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

    def record(self, step: Step, projected: Buffer, scalars: Buffer, y: Buffer) -> None:
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
            engine.record_linear(step, mixed, self.out, None, m=step.rows, n=engine.config.width, k=vs, split=0, out32=y)
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
        engine.record_linear(step, mixed, self.out, None, m=step.rows, n=engine.config.width, k=vs, split=0, out32=y)


class MatrixMemoryMixer:
    """Matrix memory with stabilised exponential input and forget gates."""

    def __init__(self, engine, spec: MatrixMemorySpec, weights, prefix: str, projection: Projection):
        self.spec, self.projection, self.prefix = spec, projection, prefix
        for name in "qkvg":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"])
        for name in "if":
            projection.add(f"{prefix}.{name}", weights[f"{prefix}.{name}"], weights[f"{prefix}.{name}.b"], fp32=True)
        self.norm = engine.upload_vector(weights[f"{prefix}.norm"])
        self.out = engine.upload_matrix(weights[f"{prefix}.o"])
        self.state_stride = matrix_state_elements(spec.heads, spec.dim, spec.vdim, normalized=True)
        self.state = engine.empty_bytes(engine.sequences.rows * self.state_stride * 4)

    def record(self, step: Step, projected: Buffer, scalars: Buffer, y: Buffer) -> None:
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
            engine.record_linear(step, mixed, self.out, None, m=step.rows, n=engine.config.width, k=vs, split=0, out32=y)
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
        engine.record_linear(step, mixed, self.out, None, m=step.rows, n=engine.config.width, k=vs, split=0, out32=y)


SINGLE_MIXERS = {AttentionSpec: AttentionMixer, DeltaSpec: DeltaMixer, MatrixMemorySpec: MatrixMemoryMixer}


class LayerMixer:
    """A layer's mixer: one, or two side by side whose normed outputs the residual norm averages."""

    def __init__(self, engine, spec, weights, prefix: str):
        self.projection = Projection()
        self.branch_norms = None
        if isinstance(spec, ParallelSpec):
            self.branches = [SINGLE_MIXERS[type(one)](engine, one, weights, f"{prefix}.{side}", self.projection)
                             for side, one in (("left", spec.left), ("right", spec.right))]
            self.branch_norms = [engine.upload_vector(weights[f"{prefix}.{side}.out"]) for side in ("left", "right")]
        else:
            self.branches = [SINGLE_MIXERS[type(spec)](engine, spec, weights, prefix, self.projection)]
        self.projection.upload(engine)

    def record(self, step: Step, x: Buffer) -> List[Buffer]:
        """Outputs of the branches."""
        projected, scalars = self.projection.record(step, x)
        outputs = [step.engine.work32(f"sublayer_{index}", step.engine.config.width) for index in range(len(self.branches))]
        for branch, y in zip(self.branches, outputs):
            branch.record(step, projected, scalars, y)
        return outputs


def attention_specs(config) -> list:
    """Attention mixers of a model in the order their layers claim cache regions."""
    found = []
    for layer in config.layers:
        branches = (layer.mixer.left, layer.mixer.right) if isinstance(layer.mixer, ParallelSpec) else (layer.mixer,)
        found += [spec for spec in branches if isinstance(spec, AttentionSpec)]
    return found

"""Prompts and decoding of models composed of sequence mixers (``model.MixerConfig``) -- the counterpart
of ``decode_engine.DecodeEngine`` for dense bfloat16 (or fp32) weights, an fp32 residual, an
unquantised row cache and recurrent matrix states, over the same runtime: dispatch lists recorded once
per shape, batches for prompts, prebaked plans (CUDA graphs with device-side token chaining) for decode.

``run`` is the one step function: it advances sequences by the given tokens, from whatever their
earlier steps left in the cache and the states, and returns logits where they are asked for.  ``prefill``,
``step`` and ``generate_chained`` (the interface of ``DecodeEngine``) and ``generate`` are built on it."""

from __future__ import annotations

import math
from collections import OrderedDict
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np

from . import parameters
from .cuda_native import Batch, Buffer, DispatchItem, Prebaked, Runtime, pack_records, sample_f32
from .feed_forward import FEED_FORWARDS
from .kv_cache import RowLayout, RowRegion, SequenceTable
from .mixers import LayerMixer, Step, attention_specs
from .model import AttentionSpec, MixerConfig
from .quantize import rotary_pairs
from .residual import RESIDUALS
from .safetensors_archive import as_bfloat16_bits, as_float32

ARGMAX_PARTS = 32


def _draw_seed(seed: int, *counters: int) -> int:
    """A well-mixed 64-bit seed per draw (splitmix64 steps): neighbouring seeds and counters share nothing."""
    mask, state = (1 << 64) - 1, seed
    for counter in (0, *counters):
        state = (state + counter + 0x9E3779B97F4A7C15) & mask
        state = ((state ^ (state >> 30)) * 0xBF58476D1CE4E5B9) & mask
        state = ((state ^ (state >> 27)) * 0x94D049BB133111EB) & mask
        state ^= state >> 31
    return state or 1
GROUP = (256, 1, 1)


class _Layer:
    """Device weights of one layer."""

    def __init__(self, engine: "MixerEngine", index: int, weights):
        layer, prefix = engine.config.layers[index], f"l{index}"
        self.index = index
        self.mixer = LayerMixer(engine, layer.mixer, weights, f"{prefix}.mix", index)
        self.feed_forward = None
        if layer.feed_forward:
            self.feed_forward = FEED_FORWARDS[type(layer.feed_forward)](engine, layer.feed_forward, weights, f"{prefix}.mlp")
        if engine.config.token_side:
            self.side_gate, self.side_proj = (engine.upload_matrix(weights[f"{prefix}.side.{name}"]) for name in ("gate", "proj"))
            self.side_norm = engine.upload_vector(weights[f"{prefix}.side.norm"])


class _Plan:
    """A recorded step of one shape with the small buffers the host writes before it runs."""

    def __init__(self, engine: "MixerEngine", sequences: int, tokens: int):
        self.sequences, self.tokens = sequences, tokens
        self.ids = engine.empty_bytes(max(sequences * tokens * 8, 16))
        self.past = engine.empty_bytes(max(sequences * 4, 16))
        self.rows = engine.empty_bytes(max(sequences * 4, 16))
        self.items: List[DispatchItem] = []
        self.step = Step(engine, sequences, tokens, self.ids, self.past, self.rows, self._run)
        # what the device buffers hold, so that a chained or repeated step does not write them again
        self.device_past: Optional[tuple] = None
        self.device_rows: Optional[tuple] = None

    def _run(self, name: str, buffers, params: bytes) -> None:
        self.items.append(DispatchItem(name, list(buffers), params, (1, 1, 1), GROUP))

    def write(self, tokens, past, rows) -> None:
        self.ids.write(0, np.asarray(tokens, np.int64).reshape(-1))
        if self.device_past != tuple(past):
            self.past.write(0, np.asarray(past, np.uint32))
        if self.device_rows != tuple(rows):
            self.rows.write(0, np.asarray(rows, np.uint32))
        self.device_past, self.device_rows = tuple(past), tuple(rows)


class MixerEngine:
    def __init__(self, runtime: Runtime, config: MixerConfig, weights, *, batch: int = 1, capacity: int = 1024,
                 sequences: Optional[int] = None, token_capacity: Optional[int] = None, page: int = 16,
                 dtype: str = "bfloat16", prompt_rows: int = 2048):
        """``batch``: sequences ``step`` decodes side by side; ``capacity``: most tokens of a sequence;
        ``sequences``: live sequences at most (default ``batch``); ``token_capacity``: token slots they
        share (default: all of them at full length); ``prompt_rows``: rows of a prompt that run at
        once, longer ones run in portions."""
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"unsupported element type: {dtype}")
        self.runtime, self.config, self.batch, self.capacity = runtime, config, batch, capacity
        self.suffix, self.itemsize = ("bf16", 2) if dtype == "bfloat16" else ("f32", 4)
        self.max_rows = max(min(prompt_rows, capacity), batch)
        rows = max(sequences or batch, batch)
        pages = lambda tokens: (tokens + page - 1) // page * page
        self.token_capacity = pages(token_capacity) if token_capacity else rows * pages(capacity)
        self.sequences = SequenceTable(rows, capacity, self.token_capacity, page)
        owners = attention_specs(config)
        self.layout = RowLayout([(spec.kv_heads, spec.dim, spec.vdim) for _, spec in owners])
        self._regions: Dict[int, List[RowRegion]] = {}  # of every layer with keys and values of its own
        for (layer, _), region in zip(owners, self.layout.regions):
            self._regions.setdefault(layer, []).append(region)
        self._claimed: Dict[int, int] = {}
        self.token_pool = self.empty_bytes(self.token_capacity * self.layout.token_elements * self.itemsize)
        self.slot_table = self.empty_bytes(rows * capacity * 4)
        self._work: Dict[tuple, Buffer] = {}
        self._trig: Dict[object, Buffer] = {}
        self._prompt_plans: "OrderedDict[int, tuple]" = OrderedDict()
        self._decode_plans: Dict[int, tuple] = {}
        self.residual = RESIDUALS[config.norm](self, weights)
        self.token_side = self.upload_matrix(weights["side.embed"]) if config.token_side else None
        self.layers = [_Layer(self, index, weights) for index in range(len(config.layers))]
        self.head = self.residual.embedding if config.tied_head else self.upload_matrix(weights["head"])
        self._lockstep = None  # rows of the sequences ``step`` decodes, once opened

    # ---- device memory --------------------------------------------------------------------------
    def empty_bytes(self, nbytes: int) -> Buffer:
        return Buffer.create(self.runtime, nbytes)

    def upload_matrix(self, array) -> Buffer:
        """A weight matrix in the model's element type."""
        return Buffer.of_array(self.runtime, as_bfloat16_bits(array) if self.itemsize == 2 else as_float32(array))

    def upload_vector(self, array) -> Buffer:
        """Norm weights, biases and the like, fp32 in every model."""
        return Buffer.of_array(self.runtime, as_float32(np.asarray(array)))

    def work(self, name: str, columns: int) -> Buffer:
        """Workspace of ``max_rows`` rows in the element type; layers of the same size share it."""
        return self._workspace(name, columns, self.itemsize)

    def work32(self, name: str, columns: int) -> Buffer:
        return self._workspace(name, columns, 4)

    def _workspace(self, name: str, columns: int, itemsize: int) -> Buffer:
        return self._workspace_bytes((name, columns, itemsize), self.max_rows * columns * itemsize)

    def rotary_table(self, rotary) -> Buffer:
        if rotary not in self._trig:
            self._trig[rotary] = Buffer.of_array(self.runtime, rotary_pairs(self.capacity, rotary))
        return self._trig[rotary]

    def scratch(self, name: str, nbytes: int) -> Buffer:
        """Workspace of another shape; users of the same name and size share it."""
        return self._workspace_bytes((name, nbytes), nbytes)

    def _workspace_bytes(self, key: tuple, nbytes: int) -> Buffer:
        if key not in self._work:
            self._work[key] = self.empty_bytes(max(nbytes, 16))
        return self._work[key]

    def attention_region(self, layer: int, spec: AttentionSpec) -> RowRegion:
        """Where a cache row holds the keys and values that an attention mixer of the layer reads."""
        if spec.kv_from is not None:
            return self._regions[spec.kv_from][0]
        place = self._claimed.get(layer, 0)
        self._claimed[layer] = place + 1
        return self._regions[layer][place]

    def cache_rows(self, region: RowRegion) -> dict:
        """Parameters of the kernels that reach into the cache."""
        return dict(token_stride=self.layout.token_elements, key_offset=region.key_offset, value_offset=region.value_offset,
                    table_stride=self.sequences.stride, table_rows=self.sequences.rows, pool_rows=self.token_capacity)

    def attention_splits(self, step: Step, spec: AttentionSpec) -> Tuple[int, Buffer]:
        """How many thread blocks share the keys of a (sequence, key/value head) when few rows ask, and
        the scratch their partial results meet in."""
        heads = step.sequences * spec.kv_heads
        visible = self.capacity
        if spec.window:
            visible = min(visible, spec.window.keep_first + spec.window.size + step.tokens - 1)
        splits = max(1, min(64, 444 // heads, (visible + 63) // 64))
        if step.tokens * (spec.heads // spec.kv_heads) > 16:
            splits = 1
        width = next((v for v in (32, 64, 128) if spec.vdim <= v), 256)
        counters = (heads * 4 + 255) // 256 * 256
        nbytes = counters + heads * splits * (32 + 16 * width) * 4
        return splits, self.scratch(f"attention_scratch_{counters}", nbytes)  # zero-filled: the arrival counters start at zero

    # ---- recording --------------------------------------------------------------------------------
    def record_linear(self, step: Step, x: Buffer, weight: Buffer, out: Optional[Buffer], *, m: int, n: int, k: int,
                      split: int, out32: Optional[Buffer] = None, bias: Optional[Buffer] = None, epilogue=None,
                      table: Optional[Buffer] = None, table_stride: int = 0, table_offset: int = 0, scale: float = 1.0) -> None:
        absent = weight
        step.run(step.element("dense_linear"),
                 [x, weight, bias or absent, out or absent, out32 or absent, step.ids, table or absent],
                 parameters.dense_linear(m=m, n=n, k=k, split=split, has_bias=bias is not None, epilogue=epilogue,
                                         table_rows=self.config.vocabulary if table else 0, table_stride=table_stride,
                                         table_offset=table_offset, scale=scale))

    def _record_layers(self, step: Step) -> None:
        """The stream of the step ends with the output of the last layer."""
        config, width = self.config, self.config.width
        step.stream = stream = self.residual.open(step)
        for layer in self.layers:
            layer.mixer.record(step)
            stream.close(branch_norms=layer.mixer.branch_norms)
            if layer.feed_forward:
                layer.feed_forward.record(step)
                stream.close()
            if config.token_side:
                dim = config.token_side.dim
                gated = self.work("token_side", dim)
                self.record_linear(step, stream.x, layer.side_gate, gated, m=step.rows, n=dim, k=width, split=dim,
                                   epilogue="token_gate", table=self.token_side, table_stride=dim * len(self.layers),
                                   table_offset=layer.index * dim)
                stream.product(gated, layer.side_proj, k=dim)
                stream.close(norm=layer.side_norm)

    def _record_logits(self, step: Step, chosen: Buffer, count: int, logits: Buffer, every: bool = False) -> None:
        """``every``: the chosen rows are all rows in order."""
        config = self.config
        rows = step.stream.chosen_rows(chosen, count, every)
        self.record_linear(step, rows, self.head, None, m=count, n=config.vocabulary, k=config.width, split=0, out32=logits,
                           scale=config.logit_scale)

    def _decode_plan(self, sequences: int):
        """(plan, graph, logits, picked tokens) of a step of one token for each of ``sequences`` sequences."""
        if sequences not in self._decode_plans:
            plan = _Plan(self, sequences, 1)
            vocabulary = self.config.vocabulary
            logits = self.empty_bytes(sequences * vocabulary * 4)
            chosen = Buffer.of_array(self.runtime, np.arange(sequences, dtype=np.uint32))
            candidates = self.empty_bytes(sequences * ARGMAX_PARTS * 8)
            picked = self.empty_bytes(max(sequences * 4, 16))
            self._record_layers(plan.step)
            self._record_logits(plan.step, chosen, sequences, logits, every=True)
            plan.step.run("llmopt_argmax_f32", [logits, candidates], parameters.u32s([sequences, vocabulary, ARGMAX_PARTS]))
            plan.step.run("llmopt_advance_tokens", [candidates, picked, plan.ids, plan.past],
                          parameters.u32s([sequences, ARGMAX_PARTS, 1]))
            graph = Prebaked(self.runtime, plan.items, plan.ids, picked)
            self._decode_plans[sequences] = (plan, graph, logits, picked)
        return self._decode_plans[sequences]

    def _prompt_plan(self, tokens: int):
        """(plan, packed dispatch list) of ``tokens`` rows of one sequence."""
        if tokens not in self._prompt_plans:
            plan = _Plan(self, 1, tokens)
            self._record_layers(plan.step)
            while len(self._prompt_plans) >= 32:
                self._prompt_plans.popitem(last=False)
            self._prompt_plans[tokens] = (plan, pack_records(plan.items))
        self._prompt_plans.move_to_end(tokens)
        return self._prompt_plans[tokens]

    # ---- the step -----------------------------------------------------------------------------------
    def open(self) -> int:
        """A new sequence with nothing behind it."""
        return self.sequences.open()

    def close(self, sequence: int) -> None:
        """Gives back what a sequence holds."""
        self.sequences.close(sequence)

    def _reserve(self, sequence: int, tokens: int) -> None:
        changed = self.sequences.reserve(sequence, tokens)
        if len(changed):
            first = sequence * self.capacity + changed.start
            self.slot_table.write(first * 4, self.sequences.table[sequence, changed.start:changed.stop])

    def run(self, entries: Sequence[tuple]) -> List[np.ndarray]:
        """One step.  ``entries``: (sequence, tokens, want) each; every sequence advances by its tokens.
        Returns per entry the fp32 logits [len(want), vocabulary] at the places ``want`` among its tokens."""
        sequences = [entry[0] for entry in entries]
        if len(set(sequences)) != len(sequences):
            raise ValueError("a sequence can only appear once in a step")
        for sequence, tokens, want in entries:
            if not self.sequences.live(sequence):
                raise ValueError("the sequence is not open")
            if len(tokens) == 0 or any(not 0 <= place < len(tokens) for place in want):
                raise ValueError("an entry needs tokens, and its places must lie among them")
            if any(not 0 <= token < self.config.vocabulary for token in tokens):
                raise ValueError("a token lies outside the vocabulary")
            if self.sequences.lengths[sequence] + len(tokens) > self.capacity:
                raise ValueError("the cache capacity is exhausted")
        if all(len(tokens) == 1 for _, tokens, _ in entries):
            return self._run_decode(entries)
        return [self._run_prompt(*entry) for entry in entries]

    def _run_decode(self, entries) -> List[np.ndarray]:
        plan, graph, logits, _ = self._decode_plan(len(entries))
        rows = [entry[0] for entry in entries]
        for row in rows:
            self._reserve(row, 1)
        past = [self.sequences.lengths[row] for row in rows]
        plan.write([entry[1][0] for entry in entries], past, rows)
        graph.execute(token=int(entries[0][1][0]), past_tokens=past[0])
        plan.device_past = tuple(p + 1 for p in past)  # advanced on the device
        for row in rows:
            self.sequences.advance(row, 1)
        vocabulary = self.config.vocabulary
        if not any(len(entry[2]) for entry in entries):
            return [np.empty((0, vocabulary), np.float32) for _ in entries]
        values = logits.to_numpy(np.float32, (len(entries), vocabulary))
        return [values[index][None, :].repeat(len(entry[2]), 0) for index, entry in enumerate(entries)]

    def _run_prompt(self, sequence: int, tokens: Sequence[int], want: Sequence[int]) -> np.ndarray:
        out = np.empty((len(want), self.config.vocabulary), np.float32)
        places = np.asarray(want, np.int64)
        for first in range(0, len(tokens), self.max_rows):
            portion = tokens[first:first + self.max_rows]
            here = np.nonzero((places >= first) & (places < first + len(portion)))[0]
            logits = self._run_portion(sequence, portion, places[here] - first)
            if logits is not None:
                out[here] = logits
        return out

    def _run_portion(self, sequence: int, tokens: Sequence[int], want: np.ndarray) -> Optional[np.ndarray]:
        plan, records = self._prompt_plan(len(tokens))
        self._reserve(sequence, len(tokens))
        plan.write(tokens, [self.sequences.lengths[sequence]], [sequence])
        commands = Batch(self.runtime)
        commands.dispatch_recorded(records)
        logits = None
        if len(want):
            logits = self.empty_bytes(len(want) * self.config.vocabulary * 4)
            chosen = Buffer.of_array(self.runtime, np.ascontiguousarray(want, np.uint32))
            kept, plan.items = plan.items, []
            self._record_logits(plan.step, chosen, len(want), logits)
            for item in plan.items:
                commands.dispatch_item(item)
            plan.items = kept
        commands.commit()
        self.sequences.advance(sequence, len(tokens))
        return None if logits is None else logits.to_numpy(np.float32, (len(want), self.config.vocabulary))

    # ---- the interface of the decode engine -------------------------------------------------------------
    def _row(self, sequence: int) -> int:
        """Row of sequence ``sequence`` of the ``batch`` that ``step`` decodes."""
        if self._lockstep is None:
            self._lockstep = [self.sequences.open() for _ in range(self.batch)]
        if not 0 <= sequence < self.batch:
            raise ValueError("no such sequence")
        return self._lockstep[sequence]

    def restart(self, sequence: int = 0) -> None:
        """Sequence ``sequence`` of the batch has nothing behind it again."""
        row = self._row(sequence)
        self.sequences.close(row)
        self._lockstep[sequence] = self.sequences.open(row)

    def prefill(self, tokens: Sequence[int], sequence: int = 0) -> int:
        """The whole prompt of one sequence of the batch from an empty cache; the first generated token."""
        self.restart(sequence)
        logits = self.run([(self._row(sequence), list(tokens), [len(tokens) - 1])])[0]
        return int(np.argmax(logits[0]))

    def step(self, tokens: Sequence[int], past_tokens: Optional[int] = None) -> List[int]:
        """One greedy step of the whole batch: token ids in, next token ids out.  ``past_tokens``, when
        given, must be what every sequence has behind it."""
        if len(tokens) != self.batch:
            raise ValueError("one token per sequence is required")
        rows = [self._row(index) for index in range(self.batch)]
        if past_tokens is not None and any(self.sequences.lengths[row] != past_tokens for row in rows):
            raise ValueError("past_tokens disagrees with the sequences")
        self.run([(row, [int(token)], []) for row, token in zip(rows, tokens)])
        return self._decode_plan(self.batch)[3].to_numpy(np.int32)[:self.batch].tolist()

    def generate_chained(self, tokens: Sequence[int], past_tokens: int, steps: int):
        """``steps`` device-chained greedy steps; returns (ids of sequence 0, device ms)."""
        rows = [self._row(index) for index in range(self.batch)]
        if len(tokens) != self.batch:
            raise ValueError("one token per sequence is required")
        if any(self.sequences.lengths[row] != past_tokens for row in rows):
            raise ValueError("past_tokens disagrees with the sequences")
        if past_tokens + steps > self.capacity:
            raise ValueError("the cache capacity is exhausted")
        plan, graph, _, _ = self._decode_plan(self.batch)
        for row in rows:
            self._reserve(row, steps)
        plan.write(tokens, [past_tokens] * self.batch, rows)
        ids, elapsed = graph.execute_chained(token=int(tokens[0]), past_tokens=past_tokens, steps=steps)
        plan.device_past = (past_tokens + steps,) * self.batch
        for row in rows:
            self.sequences.advance(row, steps)
        return ids, elapsed

    def rewind(self, past_tokens: int) -> None:
        """Declares that every sequence of the batch has ``past_tokens`` tokens behind it (measurements over a
        context that was never computed; the states keep what they hold)."""
        for index in range(self.batch):
            row = self._row(index)
            self._reserve(row, max(0, past_tokens - self.sequences.lengths[row]))
            self.sequences.lengths[row] = past_tokens

    # ---- generation ---------------------------------------------------------------------------------------
    def generate(self, prompts: Sequence[Sequence[int]], steps: int, *, temperature: float = 0.0, top_k: int = 0,
                 top_p: float = 0.0, min_p: float = 0.0, seed: int = 1, stop: Sequence[int] = ()) -> List[List[int]]:
        """Generates up to ``steps`` tokens after every prompt.  At most ``batch`` sequences are live; a
        sequence that ends (its length, or a token of ``stop``) makes room for the next prompt, and the live
        ones decode side by side whatever their lengths."""
        waiting = list(enumerate(prompts))[::-1]
        results: List[List[int]] = [[] for _ in prompts]
        live: "OrderedDict[int, int]" = OrderedDict()  # prompt -> sequence

        def pick(index: int, logits: np.ndarray) -> int:
            return sample_f32(logits, temperature=temperature, top_k=top_k, top_p=top_p, min_p=min_p,
                              seed=_draw_seed(seed, index, len(results[index])))

        def take(index: int, token: int) -> None:
            results[index].append(token)
            if len(results[index]) >= steps or token in stop:
                self.close(live.pop(index))

        if steps <= 0:
            return results
        while waiting or live:
            while waiting and len(live) < self.batch:
                index, prompt = waiting.pop()
                live[index] = self.open()
                take(index, pick(index, self.run([(live[index], list(prompt), [len(prompt) - 1])])[0][0]))
            if live:
                order = list(live)
                logits = self.run([(live[index], [results[index][-1]], [0]) for index in order])
                for index, row in zip(order, logits):
                    take(index, pick(index, row[0]))
        return results

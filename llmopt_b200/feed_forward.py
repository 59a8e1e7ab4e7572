"""Record builders of the feed-forward sublayers: dense (activation, or silu-gated) and routed experts.  Each reads the
stream's input and ends in the stream's product (``residual``)."""

from __future__ import annotations

import numpy as np

from . import parameters
from .model import ExpertsSpec, FeedForwardSpec


def _interleaved(gate: np.ndarray, up: np.ndarray) -> np.ndarray:
    """Rows of gate and up in turn: a pair of neighbouring outputs belongs together."""
    return np.stack([np.asarray(gate), np.asarray(up)], axis=1).reshape(-1, gate.shape[-1])


class DenseFeedForward:
    def __init__(self, engine, spec: FeedForwardSpec, weights, prefix: str):
        self.spec = spec
        up = weights[f"{prefix}.up"]
        self.up = engine.upload_matrix(_interleaved(weights[f"{prefix}.gate"], up) if spec.gated else up)
        self.down = engine.upload_matrix(weights[f"{prefix}.down"])

    def record(self, step) -> None:
        engine, inner = step.engine, self.spec.width
        hidden, columns = engine.work("feed_forward", inner), 2 * inner if self.spec.gated else inner
        engine.record_linear(step, step.stream.x, self.up, hidden, m=step.rows, n=columns, k=engine.config.width, split=columns,
                             epilogue="silu_pair" if self.spec.gated else self.spec.activation)
        step.stream.product(hidden, self.down, k=inner)


STREAMED_ROWS = 64  # most rows of a step whose experts' weights are streamed
EXPERT_TILE = 128  # rows of a tile of sorted rows


def route_words(rows: int, experts: int, top: int) -> int:
    """Words of a step's route (csrc/experts.cu, ``Route``): experts, their first slots, row and score per slot."""
    return 4 + (experts + 3) // 4 * 4 + (experts + 4) // 4 * 4 + 2 * rows * top


class RoutedExperts:
    """All experts' matrices as one; few rows of a bfloat16 model take the streaming kernels, others are sorted by expert."""

    def __init__(self, engine, spec: ExpertsSpec, weights, prefix: str):
        self.spec = spec
        expert = lambda index, name: weights[f"{prefix}.e{index}.{name}"]
        self.router = engine.upload_matrix(weights[f"{prefix}.router"])
        self.up = engine.upload_matrix(np.concatenate(
            [_interleaved(expert(index, "gate"), expert(index, "up")) for index in range(spec.experts)]))
        self.down = engine.upload_matrix(np.concatenate([expert(index, "down") for index in range(spec.experts)]))

    def _streams(self, step) -> bool:
        spec, engine = self.spec, step.engine
        return (engine.itemsize == 2 and step.rows <= STREAMED_ROWS and engine.config.width % 8 == 0 and spec.width % 8 == 0 and
                spec.experts <= 1024 and step.rows * spec.top <= 4096 and (3 * spec.experts + 1 + 2 * step.rows * spec.top) * 4 <= 48 * 1024)

    def record(self, step) -> None:
        engine, spec = step.engine, self.spec
        logits = engine.work32("router", spec.experts)
        engine.record_linear(step, step.stream.x, self.router, None, m=step.rows, n=spec.experts, k=engine.config.width, split=0,
                             out32=logits)
        (self._record_streamed if self._streams(step) else self._record_sorted)(step, logits)

    def _record_streamed(self, step, logits) -> None:
        engine, spec, width = step.engine, self.spec, step.engine.config.width
        rows = min(STREAMED_ROWS, engine.max_rows)
        route = engine.scratch("route", route_words(rows, spec.experts, spec.top) * 4)
        hidden = engine.scratch("experts_hidden", rows * spec.top * spec.width * engine.itemsize)
        size = dict(rows=step.rows, experts=spec.experts, top=spec.top)
        step.run("llmopt_route_step_f32", [logits, route], parameters.route(**size))
        step.run("llmopt_expert_step_bf16", [step.stream.x, self.up, route, hidden],
                 parameters.expert_step(**size, n=2 * spec.width, k=width))
        step.run("llmopt_expert_step_residual_bf16", [hidden, self.down, route, *step.stream.ending],
                 parameters.expert_step(**size, n=width, k=spec.width))

    def _record_sorted(self, step, logits) -> None:
        engine, spec, width = step.engine, self.spec, step.engine.config.width
        most, pairs = engine.max_rows * spec.top, step.rows * spec.top
        chosen, scores, row_of_slot, score_of_slot, slot_of_pair = (
            engine.scratch(name, most * 4) for name in ("chosen", "scores", "row_of_slot", "score_of_slot", "slot_of_pair"))
        plan = engine.scratch("expert_plan", 16 * (1 + most // EXPERT_TILE + min(spec.experts, most)))
        x, hidden = engine.scratch("experts_x", most * width * engine.itemsize), engine.scratch(
            "experts_sorted", most * spec.width * engine.itemsize)
        y = engine.scratch("experts_y", most * width * 4)
        size = dict(rows=step.rows, experts=spec.experts, top=spec.top)
        step.run("llmopt_route_rows_f32", [logits, chosen, scores], parameters.route(**size))
        step.run("llmopt_route_plan", [chosen, scores, plan, row_of_slot, score_of_slot, slot_of_pair], parameters.route(**size))
        step.run(step.element("gather_rows"), [step.stream.x, row_of_slot, x],
                 parameters.gather_rows(count=pairs, source_rows=step.rows, width=width))
        step.run(step.element("expert_rows"), [x, self.up, plan, score_of_slot, hidden],
                 parameters.expert_rows(pairs=pairs, n=2 * spec.width, k=width, experts=spec.experts, paired=True))
        step.run(step.element("expert_rows"), [hidden, self.down, plan, score_of_slot, y],
                 parameters.expert_rows(pairs=pairs, n=width, k=spec.width, experts=spec.experts, paired=False))
        step.run(step.element("expert_combine"), [y, slot_of_pair, *step.stream.ending],
                 parameters.expert_combine(rows=step.rows, width=width, top=spec.top))


FEED_FORWARDS = {FeedForwardSpec: DenseFeedForward, ExpertsSpec: RoutedExperts}

"""The residual streams of the sequence-mixer models: what surrounds the sublayers.

A residual owns the embedding table and the norms on the device.  ``open`` starts a stream for one recorded step: the
stream records the embedding, hands every sublayer its input (``x``), takes the product that ends the sublayer
(``product``, once per branch) and, after ``close``, has the next sublayer's input.  ``chosen_rows`` are the inputs of the output
projection."""

from __future__ import annotations

import numpy as np

from . import parameters
from .cuda_native import Buffer
from .model import MixerConfig, sublayer_norms
from .safetensors_archive import as_float32


class PostNormResidual:
    """x <- x + norm(sublayer(x)): the sublayers read the residual itself, and their fp32 outputs are RMS-normed (two
    branches: averaged after a norm each) in a row kernel of their own."""

    def __init__(self, engine, weights):
        config: MixerConfig = engine.config
        self.engine = engine
        self.embedding = engine.upload_matrix(weights["embed"])
        self.norms = [engine.upload_vector(weights[name]) for (name,) in sublayer_norms(config)]
        self.final_norm = engine.upload_vector(weights["final.norm"])

    def open(self, step):
        return _PostNormStream(self, step)


class _PostNormStream:
    def __init__(self, residual: PostNormResidual, step):
        engine, width = residual.engine, residual.engine.config.width
        self.residual, self.step, self.sublayer, self.current = residual, step, 0, 0
        self.rows = [engine.work32("residual_a", width), engine.work32("residual_b", width)]
        self.copies = self.rows if engine.itemsize == 4 else [engine.work("copy_a", width), engine.work("copy_b", width)]
        step.run(step.element("embedding_residual"), [step.ids, residual.embedding, self.rows[0], self.copies[0]],
                 parameters.embedding(tokens=step.rows, vocabulary=engine.config.vocabulary, width=width))

    @property
    def x(self) -> Buffer:
        return self.copies[self.current]

    def _output(self, branch: int) -> Buffer:
        return self.residual.engine.work32(f"sublayer_{branch}", self.residual.engine.config.width)

    def product(self, x: Buffer, weight: Buffer, *, k: int, bias=None, branch: int = 0) -> None:
        engine = self.residual.engine
        engine.record_linear(self.step, x, weight, None, m=self.step.rows, n=engine.config.width, k=k, split=0,
                             out32=self._output(branch), bias=bias)

    def close(self, norm=None, branch_norms=None) -> None:
        """Ends a sublayer: its own norm, or the given one (with no offset)."""
        config, step = self.residual.engine.config, self.step
        offset = config.norm_offset
        if norm is None:
            norm = self.residual.norms[self.sublayer]
            self.sublayer += 1
        else:
            offset = 0.0
        left, right = branch_norms or (norm, norm)
        step.run(step.element("residual_norm"),
                 [self.rows[self.current], self._output(0), norm, self._output(1) if branch_norms else self._output(0), left,
                  right, self.rows[1 - self.current], self.copies[1 - self.current]],
                 parameters.residual_norm(rows=step.rows, width=config.width, epsilon=config.epsilon, weight_offset=offset,
                                          pair=bool(branch_norms)))
        self.current = 1 - self.current

    def chosen_rows(self, chosen: Buffer, count: int, every: bool) -> Buffer:
        engine, step = self.residual.engine, self.step
        normed = engine.work("final_normed", engine.config.width)
        step.run(step.element("gather_norm"), [self.rows[self.current], chosen, self.residual.final_norm, normed],
                 parameters.gather_norm(count=count, source_rows=step.rows, width=engine.config.width,
                                        epsilon=engine.config.epsilon, weight_offset=engine.config.norm_offset))
        return normed


class TanhResidual:
    """x <- x + post(sublayer(pre(x))) with norms tanh(alpha x) weight + bias.  They need no statistics of the row, so both
    norms and the residual add ride in the writeback of the product that ends the sublayer, and the stream
    keeps the fp32 residual and the next sublayer's normed input."""

    def __init__(self, engine, weights):
        config: MixerConfig = engine.config
        self.engine = engine
        self.embedding = engine.upload_matrix(weights["embed"])

        def upload(name):  # weight, bias, alpha as one vector
            return engine.upload_vector(np.concatenate(
                [as_float32(np.asarray(weights[part])).reshape(-1) for part in (name, f"{name}.b", f"{name}.alpha")]))

        around = [(upload(before), upload(after)) for before, after in sublayer_norms(config)]
        # the norm ahead of every sublayer, then that of the output
        self.before = [before for before, _ in around] + [upload("final.norm")]
        self.after = [after for _, after in around]
        pairs = np.arange((config.width + 1) // 2, dtype=np.float64)
        self.turns = Buffer.of_array(engine.runtime, 10000.0 ** (-2.0 * pairs / config.width) / (2.0 * np.pi))  # per position

    def open(self, step):
        return _TanhStream(self, step)


class _TanhStream:
    def __init__(self, residual: TanhResidual, step):
        engine, config = residual.engine, residual.engine.config
        self.residual, self.step, self.sublayer = residual, step, 0
        self.rows, self.x = engine.work32("residual", config.width), engine.work("normed", config.width)
        step.run(step.element("embedding_sinusoid"),
                 [step.ids, residual.embedding, step.past, residual.turns, residual.before[0], self.rows, self.x],
                 parameters.embedding_sinusoid(rows=step.rows, tokens=step.tokens, vocabulary=config.vocabulary,
                                               width=config.width))

    @property
    def ending(self) -> list:
        """What ends a sublayer: its norm, the following one, the residual and where the following input goes."""
        return [self.residual.after[self.sublayer], self.residual.before[self.sublayer + 1], self.rows, self.x]

    def product(self, x: Buffer, weight: Buffer, *, k: int, bias=None, branch: int = 0) -> None:
        step, width = self.step, self.residual.engine.config.width
        step.run(step.element("dense_residual"), [x, weight, bias or weight, *self.ending],
                 parameters.dense_residual(m=step.rows, n=width, k=k, has_bias=bias is not None))

    def close(self, norm=None, branch_norms=None) -> None:
        self.sublayer += 1

    def chosen_rows(self, chosen: Buffer, count: int, every: bool) -> Buffer:
        if every:
            return self.x
        engine, step = self.residual.engine, self.step
        rows = engine.work("final_normed", engine.config.width)
        step.run(step.element("gather_rows"), [self.x, chosen, rows],
                 parameters.gather_rows(count=count, source_rows=step.rows, width=engine.config.width))
        return rows


RESIDUALS = {"rms": PostNormResidual, "tanh": TanhResidual}

"""The Bizodra design: its config.json and the names of its tensors, as a ``MixerConfig``.

Layers of three kinds -- matrix memory ("mlstm", "mlstm_2") and sink attention beside a gated delta rule
("parallel") -- each followed by an erf-gelu feed-forward and a gated per-layer token input.  Every
sublayer reads the residual itself and its output is normed before it is added."""

from __future__ import annotations

from .model import (AttentionSpec, DeltaSpec, FeedForwardSpec, MatrixMemorySpec, MixerConfig, MixerLayer, ParallelSpec,
                    RotarySpec, TokenSideSpec, YarnSpec, register_architecture)


def _rotary(rot: dict) -> RotarySpec:
    scaling = rot.get("scaling")
    return RotarySpec(dims=int(rot["dims"]), base=float(rot["base"]),
                      scaling=None if not scaling else YarnSpec(
                          factor=float(scaling["factor"]), original=float(scaling["original"]),
                          fast=float(scaling["fast"]), slow=float(scaling["slow"])))


def _attention(size: dict) -> AttentionSpec:
    return AttentionSpec(heads=int(size["heads"]), kv_heads=int(size["kv_heads"]), dim=int(size["dim"]),
                         vdim=int(size["vdim"]), scale=float(size["scale"]), rotary=_rotary(size["rot"]),
                         bias=True, head_norm=True, sink=True)


def _delta(size: dict) -> DeltaSpec:
    return DeltaSpec(heads=int(size["heads"]), kv_heads=int(size["kv_heads"]), dim=int(size["dim"]),
                     vdim=int(size["vdim"]), taps=int(size["conv"]))


def _matrix_memory(size: dict) -> MatrixMemorySpec:
    return MatrixMemorySpec(heads=int(size["heads"]), dim=int(size["dim"]), vdim=int(size["vdim"]),
                            gate_cap=float(size["gate_cap"]))


def _parallel(size: dict) -> ParallelSpec:
    return ParallelSpec(left=_attention(size["left"]), right=_delta(size["right"]))


MIXERS = {"mlstm": _matrix_memory, "mlstm_2": _matrix_memory, "parallel": _parallel}


def _feed_forward(mlp):
    if not mlp:
        return None
    if mlp["kind"] != "dense":
        raise ValueError(f"unsupported feed-forward kind: {mlp['kind']}")
    return FeedForwardSpec(width=int(mlp["ff"]), activation="gelu")


@register_architecture("Bizodra")
def parse(config: dict) -> MixerConfig:
    layers = []
    for entry in config["layers"]:
        if entry["type"] not in MIXERS:
            raise ValueError(f"unsupported layer type: {entry['type']}")
        layers.append(MixerLayer(mixer=MIXERS[entry["type"]](entry["mixer"]), feed_forward=_feed_forward(entry.get("mlp"))))
    side = config.get("token_side")
    return MixerConfig(
        name="bizodra", width=int(config["width"]), vocabulary=int(config["vocab"]), layers=tuple(layers),
        epsilon=float(config["norm"]["eps"]), norm_offset=1.0,
        token_side=TokenSideSpec(dim=int(side["dim"])) if side else None)

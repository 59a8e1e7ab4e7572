"""The Dalorax design: its config.json and the names of its tensors, as a ``MixerConfig``.

Attention over a sliding window that keeps the sequence's first tokens, without rotation (positions are added to the
embedding), with capped scores and gated read-outs; a layer may read an earlier layer's keys and values.  Dense or routed
silu-gated feed-forward layers.  Tanh norms before and after every sublayer; the embedding table is the output
projection too."""

from __future__ import annotations

from .model import AttentionSpec, ExpertsSpec, FeedForwardSpec, MixerConfig, MixerLayer, WindowSpec, register_architecture


def _attention(size: dict) -> AttentionSpec:
    mask, softcap, source = size.get("mask"), size.get("softcap"), size.get("kv_from")
    return AttentionSpec(
        heads=int(size["heads"]), kv_heads=int(size["kv_heads"]), dim=int(size["dim"]), vdim=int(size["vdim"]),
        scale=float(size["scale"]), gate=True, weights32=True, softcap=float(softcap) if softcap else None,
        window=WindowSpec(size=int(mask["size"]), keep_first=int(mask.get("keep_first", 0))) if mask else None,
        kv_from=None if source is None else int(source))


def _feed_forward(mlp):
    if not mlp:
        return None
    if mlp["kind"] == "dense":
        return FeedForwardSpec(width=int(mlp["ff"]), activation="silu", gated=True)
    if mlp["kind"] == "moe":
        return ExpertsSpec(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), width=int(mlp["expert"]["ff"]))
    raise ValueError(f"unsupported feed-forward kind: {mlp['kind']}")


@register_architecture("Dalorax")
def parse(config: dict) -> MixerConfig:
    layers = []
    for entry in config["layers"]:
        if entry["type"] != "attention":
            raise ValueError(f"unsupported layer type: {entry['type']}")
        layers.append(MixerLayer(mixer=_attention(entry["mixer"]), feed_forward=_feed_forward(entry.get("mlp"))))
    return MixerConfig(
        name="dalorax", width=int(config["width"]), vocabulary=int(config["vocab"]), layers=tuple(layers),
        epsilon=float(config["norm"]["eps"]), norm="tanh", sinusoid=True, tied_head=True,
        logit_scale=float(config["logit_scale"]))

"""Shapes and synthetic weights of the decoder families the hot path serves:
Llama-style blocks (RMSNorm, fused QKV, RoPE, GQA attention over the Q8 cache,
SwiGLU FFN) and LFM-style gated short-conv blocks (lib/lfm25.ml:18-34).  The
weights are random-init and quantised W4A16 group-64; there is no checkpoint
loader for them here — a compiled package brings its own tensors.

The second part describes decoders composed of sequence mixers (attention over
unquantised cache rows, gated delta rule, matrix memory, two of them side by side) and
dense or routed feed-forward layers with bfloat16 weights, which are read from a folder with a config.json and a
safetensors checkpoint: ``ARCHITECTURES`` maps the config's architecture name to the
function that reads it."""

from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass, field
from typing import Callable, Dict, Optional, Sequence, Tuple, Union

import numpy as np

from .quantize import pack_int4_weight


@dataclass(frozen=True)
class ModelConfig:
    name: str
    hidden: int
    layers: Sequence[str]          # "attention" or "conv" per block
    query_heads: int
    kv_heads: int
    head_dim: int
    intermediate: int
    vocabulary: int
    epsilon: float = 1e-5
    rope_theta: float = 1e5
    kv_group_size: int = 64

    @property
    def attention_layers(self) -> int:
        return sum(1 for kind in self.layers if kind == "attention")

    @property
    def conv_layers(self) -> int:
        return sum(1 for kind in self.layers if kind == "conv")


SMOLLM2_135M = ModelConfig("smollm2-135m-shaped", 576, ("attention",) * 30, 9, 3, 64, 1536, 49152, 1e-5, 1e5)
# lib/lfm25.ml:30-33: conv and attention blocks interleaved, 10 conv + 6 attention
LFM25_350M = ModelConfig(
    "lfm2.5-350m-shaped", 1024,
    ("conv", "conv", "attention", "conv", "conv", "attention", "conv", "conv", "attention", "conv", "attention",
     "conv", "attention", "conv", "attention", "conv"),
    16, 8, 64, 4608, 65536, 1e-5, 1e6)
LLAMA3_8B = ModelConfig("llama-3-8b-shaped", 4096, ("attention",) * 32, 32, 8, 128, 14336, 128256, 1e-5, 5e5)


def tiny_config(layers=("attention", "attention"), hidden=192, heads=3, kv_heads=1, head_dim=64, intermediate=384,
                vocabulary=1024) -> ModelConfig:
    return ModelConfig("tiny", hidden, tuple(layers), heads, kv_heads, head_dim, intermediate, vocabulary, 1e-5, 1e5)


def _quantized(rng, n, k, std, fast):
    if fast:
        # uniform random nibbles and scales: same bytes-per-weight, no host quantisation pass
        packed = rng.integers(0, 256, size=(n, k // 2), dtype=np.uint8)
        scale = rng.uniform(0.5 * std / 7 * 3, 1.5 * std / 7 * 3, size=(n, k // 64)).astype(np.float16)
        return packed, scale
    return pack_int4_weight((rng.standard_normal((n, k)) * std).astype(np.float32))


def random_weights(config: ModelConfig, seed: int = 0, std: float = 0.02, fast: bool = False) -> dict:
    """Random-init N(0, std) weights quantised with the reference quantiser.
    ``fast`` draws packed bytes and scales directly (for multi-GB models)."""
    rng = np.random.default_rng(seed)
    hidden, dim = config.hidden, config.head_dim
    weights = {}
    embedding = (rng.standard_normal((config.vocabulary, hidden)) * std).astype(np.float32)
    weights["embedding"] = embedding.astype(np.float16)
    if fast:
        weights["lm_head"] = _quantized(rng, config.vocabulary, hidden, std, True)
    else:
        weights["lm_head"] = pack_int4_weight(embedding)  # tied embeddings: W4 copy of the table
    weights["final_norm"] = np.ones(hidden, np.float16)
    for index, kind in enumerate(config.layers):
        layer = {"input_norm": np.ones(hidden, np.float16), "ffn_norm": np.ones(hidden, np.float16)}
        if kind == "attention":
            layer["q"] = _quantized(rng, config.query_heads * dim, hidden, std, fast)
            layer["k"] = _quantized(rng, config.kv_heads * dim, hidden, std, fast)
            layer["v"] = _quantized(rng, config.kv_heads * dim, hidden, std, fast)
            layer["o"] = _quantized(rng, hidden, config.query_heads * dim, std, fast)
        else:
            layer["in_proj"] = _quantized(rng, 3 * hidden, hidden, std, fast)
            layer["conv"] = (rng.standard_normal((hidden, 1, 3)) * 0.5).astype(np.float16)
            layer["out_proj"] = _quantized(rng, hidden, hidden, std, fast)
        layer["gate"] = _quantized(rng, config.intermediate, hidden, std, fast)
        layer["up"] = _quantized(rng, config.intermediate, hidden, std, fast)
        layer["down"] = _quantized(rng, hidden, config.intermediate, std, fast)
        weights[f"layer{index}"] = layer
    return weights


def decode_bytes_per_token(config: ModelConfig, batch: int, past: int) -> dict:
    """Algorithmic bytes one decode step must move: every weight matrix and scale
    once, the KV of every sequence once, activations negligible but counted for
    the linears (x once, y once per op)."""
    hidden, dim = config.hidden, config.head_dim

    def linear(n, k):
        return n * k // 2 + n * (k // 64) * 2 + batch * k * 2 + batch * n * 2

    weights = 0
    for kind in config.layers:
        if kind == "attention":
            weights += linear((config.query_heads + 2 * config.kv_heads) * dim, hidden)
            weights += linear(hidden, config.query_heads * dim)
        else:
            weights += linear(3 * hidden, hidden) + linear(hidden, hidden)
        weights += 2 * linear(config.intermediate, hidden) + linear(hidden, config.intermediate)
    weights += linear(config.vocabulary, hidden)
    kv_per_token = 2 * config.kv_heads * dim + 2 * 2 * config.kv_heads * dim // config.kv_group_size
    attention = config.attention_layers * batch * (past * (kv_per_token + 4))
    return {"weights": weights, "attention": attention, "total": weights + attention + hidden * 2 * batch}


# ---- decoders composed of sequence mixers --------------------------------------------------------------

@dataclass(frozen=True)
class YarnSpec:
    """Frequencies of slow pairs divided by ``factor``, those of fast pairs kept, a linear ramp between."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    """The first ``dims`` dimensions of a head turn, in pairs of neighbours (2i, 2i + 1)."""

    dims: int
    base: float
    scaling: Optional[YarnSpec] = None


@dataclass(frozen=True)
class WindowSpec:
    """A token sees the last ``size`` tokens (itself included) and the first ``keep_first`` of the sequence."""

    size: int
    keep_first: int = 0


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotarySpec] = None
    bias: bool = False       # on q, k, v and the output projection
    head_norm: bool = False  # RMS norm of every query and key head before rotation
    sink: bool = False       # one more term exp(0) in the softmax denominator
    window: Optional[WindowSpec] = None
    softcap: Optional[float] = None  # score <- softcap * tanh(score / softcap)
    gate: bool = False               # read-outs times the sigmoid of a projection of the mixer's input
    kv_from: Optional[int] = None    # no keys and values of its own: those of that (earlier) layer
    weights32: bool = False          # softmax weights are not rounded to bfloat16 before they meet the values

    @property
    def prepared(self) -> bool:
        """Whether queries and keys change between projection and scores."""
        return self.head_norm or self.rotary is not None


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class MatrixMemorySpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same input; the mean of their outputs, each RMS-normed."""

    left: Union[AttentionSpec, DeltaSpec, MatrixMemorySpec]
    right: Union[AttentionSpec, DeltaSpec, MatrixMemorySpec]


@dataclass(frozen=True)
class FeedForwardSpec:
    """down(activation(up x)), or, with ``gated``, down(silu(gate x) * up x)."""

    width: int
    activation: str = "gelu"
    gated: bool = False


@dataclass(frozen=True)
class ExpertsSpec:
    """Routed gated feed-forward layers: a token goes through the ``top`` of ``experts`` with the largest scores (sigmoid of
    the router's logits); a score, not renormalised, multiplies its expert's input, and the outputs are added."""

    experts: int
    top: int
    width: int


@dataclass(frozen=True)
class TokenSideSpec:
    """Per-layer token input: a table row of ``dim`` per layer, gated by the residual."""

    dim: int


@dataclass(frozen=True)
class MixerLayer:
    mixer: Union[AttentionSpec, DeltaSpec, MatrixMemorySpec, ParallelSpec]
    feed_forward: Union[None, FeedForwardSpec, ExpertsSpec]

    @property
    def mixers(self) -> tuple:
        return (self.mixer.left, self.mixer.right) if isinstance(self.mixer, ParallelSpec) else (self.mixer,)


@dataclass(frozen=True)
class MixerConfig:
    """With ``norm`` "rms": x <- x + norm(mixer(x)), x <- x + norm(ff(x)), x <- x + norm(token side(x)) per layer; the
    sublayer norms are RMS norms that multiply by ``norm_offset`` + weight.

    With ``norm`` "tanh" every sublayer has a norm before and one after it, x <- x + post(sublayer(pre(x))), and a norm is
    tanh(alpha x) weight + bias."""

    name: str
    width: int
    vocabulary: int
    layers: Tuple[MixerLayer, ...]
    epsilon: float
    norm_offset: float = 0.0
    token_side: Optional[TokenSideSpec] = None
    norm: str = "rms"
    sinusoid: bool = False      # sinusoidal positions are added to the embedding
    tied_head: bool = False     # the embedding table is the output projection too
    logit_scale: float = 1.0

    def __post_init__(self):
        if self.width <= 0 or self.vocabulary <= 0 or not self.layers:
            raise ValueError("a model needs a width, a vocabulary and layers")
        if self.norm not in ("rms", "tanh"):
            raise ValueError(f"unsupported norm: {self.norm}")
        if self.sinusoid != (self.norm == "tanh"):
            raise ValueError("sinusoidal positions come with tanh norms, and those with sinusoidal positions")
        for index, layer in enumerate(self.layers):
            feed_forward = layer.feed_forward
            if self.norm == "tanh" and (self.token_side or isinstance(layer.mixer, ParallelSpec)):
                raise ValueError("tanh norms take single mixers and no token side input")
            if isinstance(feed_forward, ExpertsSpec):
                if self.norm != "tanh":
                    raise ValueError("routed experts come with tanh norms")
                if not 0 < feed_forward.top <= feed_forward.experts or feed_forward.width <= 0:
                    raise ValueError("a token needs at least one expert and at most all of them")
            for mixer in layer.mixers:
                kv_heads = getattr(mixer, "kv_heads", mixer.heads)
                if min(mixer.heads, kv_heads, mixer.dim, mixer.vdim) <= 0 or mixer.heads % kv_heads:
                    raise ValueError("query heads must come in whole groups per key/value head")
                if not isinstance(mixer, AttentionSpec):
                    continue
                if mixer.rotary and (mixer.rotary.dims % 2 or mixer.rotary.dims > mixer.dim):
                    raise ValueError("rotated dimensions come in pairs inside the head")
                if mixer.window and (mixer.window.size <= 0 or mixer.window.keep_first < 0):
                    raise ValueError("a window sees at least the token itself")
                if mixer.kv_from is not None:
                    source = self.layers[mixer.kv_from].mixer if 0 <= mixer.kv_from < index else None
                    if not isinstance(source, AttentionSpec) or source.kv_from is not None:
                        raise ValueError("keys and values can be shared with an earlier attention layer that has its own")
                    if (source.kv_heads, source.dim, source.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                        raise ValueError("layers that share keys and values need equal key and value heads")


ARCHITECTURES: Dict[str, Callable[[dict], MixerConfig]] = {}
# the module that registers each architecture, imported when it is first asked for
ARCHITECTURE_MODULES = {"Bizodra": "bizodra", "Dalorax": "dalorax"}


def register_architecture(name: str):
    def register(parse):
        ARCHITECTURES[name] = parse
        return parse
    return register


def parse_config(config: dict) -> MixerConfig:
    name = config.get("architecture")
    if name in ARCHITECTURE_MODULES:
        importlib.import_module("." + ARCHITECTURE_MODULES[name], __package__)
    if name not in ARCHITECTURES:
        raise ValueError(f"unsupported architecture: {name}")
    return ARCHITECTURES[name](config)


def load_model(folder: str):
    """(configuration, weights) of a folder with config.json and model.safetensors."""
    from .safetensors_archive import Archive

    with open(os.path.join(folder, "config.json")) as source:
        config = parse_config(json.load(source))
    return config, Archive(os.path.join(folder, "model.safetensors"))


def kernel_family(config: MixerConfig) -> str:
    """The smallest family of kernels (``_build.FAMILIES``) that serves a model."""
    attention = all(isinstance(mixer, AttentionSpec) for layer in config.layers for mixer in layer.mixers)
    return "attention" if attention else "mixers"


def sublayer_norms(config: MixerConfig) -> list:
    """Tensor names of the norms of every sublayer in order: (before, after) with tanh norms, (after,) with RMS norms."""
    names = []
    for index, layer in enumerate(config.layers):
        for place in (1, 2) if layer.feed_forward else (1,):
            name = f"l{index}.norm{place}"
            names.append((name, f"{name}b") if config.norm == "tanh" else (name,))
    return names


def mixer_tensors(config: MixerConfig) -> Dict[str, tuple]:
    """Name and shape of every tensor of a checkpoint."""
    width, shapes = config.width, {}
    shapes["embed"] = (config.vocabulary, width)
    if config.token_side:
        shapes["side.embed"] = (config.vocabulary, len(config.layers) * config.token_side.dim)

    def mixer(prefix, spec):
        if isinstance(spec, ParallelSpec):
            for side, one in (("left", spec.left), ("right", spec.right)):
                mixer(f"{prefix}.{side}", one)
                shapes[f"{prefix}.{side}.out"] = (width,)
            return
        heads, kv_heads = spec.heads, getattr(spec, "kv_heads", spec.heads)
        query_heads = kv_heads if isinstance(spec, DeltaSpec) else heads
        value_heads = heads if isinstance(spec, DeltaSpec) else kv_heads
        shared = isinstance(spec, AttentionSpec) and spec.kv_from is not None
        for name, rows in (("q", query_heads * spec.dim), ("k", kv_heads * spec.dim), ("v", value_heads * spec.vdim)):
            if name == "q" or not shared:
                shapes[f"{prefix}.{name}"] = (rows, width)
        shapes[f"{prefix}.o"] = (width, heads * spec.vdim)
        if not isinstance(spec, AttentionSpec) or spec.gate:
            shapes[f"{prefix}.g"] = (heads * spec.vdim, width)
        if isinstance(spec, AttentionSpec):
            if spec.bias:
                for name in "qo" if shared else "qkvo":
                    shapes[f"{prefix}.{name}.b"] = shapes[f"{prefix}.{name}"][:1]
            if spec.head_norm:
                for name in "q" if shared else "qk":
                    shapes[f"{prefix}.{name}.norm"] = (spec.dim,)
            return
        if isinstance(spec, DeltaSpec):
            for name in "qkv":
                shapes[f"{prefix}.{name}.conv"] = (shapes[f"{prefix}.{name}"][0], spec.taps)
            shapes[f"{prefix}.b"] = shapes[f"{prefix}.a"] = (heads, width)
            shapes[f"{prefix}.A_log"] = shapes[f"{prefix}.dt_bias"] = (heads,)
            shapes[f"{prefix}.norm"] = (spec.vdim,)
        else:
            shapes[f"{prefix}.norm"] = (heads * spec.vdim,)
            for name in "if":
                shapes[f"{prefix}.{name}"] = (heads, width)
                shapes[f"{prefix}.{name}.b"] = (heads,)

    def gated(prefix, inner):
        shapes[f"{prefix}.gate"] = shapes[f"{prefix}.up"] = (inner, width)
        shapes[f"{prefix}.down"] = (width, inner)

    def norm(*names):
        for name in names:
            shapes[name] = (width,)
            if config.norm == "tanh":
                shapes[f"{name}.b"], shapes[f"{name}.alpha"] = (width,), ()

    around = iter(sublayer_norms(config))
    for index, layer in enumerate(config.layers):
        norm(*next(around))
        mixer(f"l{index}.mix", layer.mixer)
        feed_forward, prefix = layer.feed_forward, f"l{index}.mlp"
        if feed_forward:
            norm(*next(around))
        if isinstance(feed_forward, ExpertsSpec):
            shapes[f"{prefix}.router"] = (feed_forward.experts, width)
            for expert in range(feed_forward.experts):
                gated(f"{prefix}.e{expert}", feed_forward.width)
        elif feed_forward and feed_forward.gated:
            gated(prefix, feed_forward.width)
        elif feed_forward:
            shapes[f"{prefix}.up"] = (feed_forward.width, width)
            shapes[f"{prefix}.down"] = (width, feed_forward.width)
        if config.token_side:
            shapes[f"l{index}.side.gate"] = (config.token_side.dim, width)
            shapes[f"l{index}.side.proj"] = (width, config.token_side.dim)
            shapes[f"l{index}.side.norm"] = (width,)
    norm("final.norm")
    if not config.tied_head:
        shapes["head"] = (config.vocabulary, width)
    return shapes


def random_mixer_weights(config: MixerConfig, seed: int = 0, std: float = 0.02, fast: bool = False) -> Dict[str, np.ndarray]:
    """Random-init weights under the checkpoint's names, as bfloat16 bits; matrices N(0, std), norm weights
    near the value that leaves a vector as it is, decays of a few to a few hundred tokens.  ``fast`` draws
    the bits of matrices directly (magnitudes 1/64 .. 1/32, for multi-GB models).  An embedding that positions are added
    to has their magnitude, so that tokens differ and take different experts."""
    from .safetensors_archive import as_bfloat16_bits

    rng = np.random.default_rng(seed)
    weights = {}
    for name, shape in mixer_tensors(config).items():
        leaf = name.rsplit(".", 1)[-1]
        offset = config.norm_offset if leaf in ("norm1", "norm2") or name == "final.norm" else 0.0
        if leaf == "alpha":
            value = rng.uniform(0.4, 0.8, size=shape)
        elif leaf in ("norm1", "norm2", "norm1b", "norm2b", "norm", "out"):
            value = rng.uniform(0.8, 1.2, size=shape) - offset
        elif leaf == "A_log":
            value = np.log(rng.uniform(1.0, 8.0, size=shape))
        elif leaf == "dt_bias":
            value = np.log(np.expm1(np.exp(rng.uniform(np.log(1e-3), np.log(0.1), size=shape))))
        elif name.endswith(".f.b"):
            value = rng.uniform(3.0, 6.0, size=shape)
        elif leaf == "conv":
            value = rng.standard_normal(shape) * 0.5
        elif leaf == "b" and len(shape) == 1:
            value = rng.standard_normal(shape) * 0.1
        elif name == "embed" and config.sinusoid:
            value = rng.standard_normal(shape, dtype=np.float32)
        elif fast:
            bits = np.frombuffer(rng.bytes(2 * int(np.prod(shape))), np.uint16)
            weights[name] = ((bits & 0x807F) | 0x3C80).reshape(shape)
            continue
        else:
            value = rng.standard_normal(shape, dtype=np.float32) * np.float32(std)
        weights[name] = as_bfloat16_bits(np.asarray(value, np.float32))
    return weights

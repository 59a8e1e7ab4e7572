"""Small configurations and random weights of the sequence-mixer models for the tests."""

import numpy as np

from llmopt_b200.model import mixer_tensors, parse_config


def memory_layer(heads=3, dim=40, vdim=24, gate_cap=6.0, ff=112, kind="mlstm"):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def parallel_layer(heads=6, kv_heads=3, dim=24, vdim=40, rot=None, scale=0.3, right=None, ff=80):
    rot = rot or {"base": 5000.0, "dims": 16, "scaling": {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}}
    right = right or {"heads": 4, "kv_heads": 2, "dim": 36, "vdim": 44, "conv": 3}
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale},
                      "right": right},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config_of(layers, width=104, vocab=150, eps=1e-5, side=24):
    return {"architecture": "Bizodra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "token_side": {"dim": side}}


def window_layer(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.4, softcap=5.0, size=9, keep_first=3, kv_from=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
             "mask": None if size is None else {"size": size, "keep_first": keep_first}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def dense_mlp(ff):
    return {"kind": "dense", "ff": ff}


def routed_mlp(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def sandwich_config(layers, width=104, vocab=150, logit_scale=0.7):
    return {"architecture": "Dalorax", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": 1e-5},
            "logit_scale": logit_scale}


def bf16_round(array):
    bits = np.ascontiguousarray(array, np.float32).view(np.uint32)
    return (((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def weights_of(config, seed=0):
    """fp32 arrays whose values are exact in bfloat16; every norm, gate and bias differs from the neutral value."""
    rng = np.random.default_rng(seed)
    out, shapes = {}, mixer_tensors(parse_config(config))
    for name, shape in shapes.items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "alpha":
            value = rng.uniform(0.3, 0.9, size=shape)
        elif f"{name}.alpha" in shapes:
            value = rng.uniform(0.6, 1.5, size=shape) * rng.choice([-1, 1], size=shape)
        elif leaf == "router":
            value = rng.standard_normal(shape) * 2.0 / np.sqrt(shape[-1])
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            value = rng.uniform(-0.4, 0.4, size=shape)
        elif leaf in ("norm", "out"):
            value = rng.uniform(0.6, 1.5, size=shape)
        elif leaf == "A_log":
            value = np.log(rng.uniform(0.5, 6.0, size=shape))
        elif leaf == "dt_bias":
            value = rng.uniform(-5.0, -1.0, size=shape)
        elif name.endswith(".f.b"):
            value = rng.uniform(1.0, 5.0, size=shape)
        elif leaf == "b" and len(shape) == 1:
            # a large constant part of a router's input would favour the same experts everywhere
            value = rng.standard_normal(shape) * (0.05 if config["architecture"] == "Dalorax" else 0.3)
        elif leaf == "conv":
            value = rng.standard_normal(shape) * 0.5
        elif name in ("embed", "side.embed"):
            value = rng.standard_normal(shape) * (3.0 if config["architecture"] == "Dalorax" else 1.0)
        else:
            value = rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = bf16_round(value)
    return out


MODELS = {
    # heads, sizes, rotated share, scale and taps all different from one another
    "mixed": config_of([memory_layer(), parallel_layer(), memory_layer(heads=2, dim=16, vdim=72, gate_cap=2.5, ff=None,
                                                                      kind="mlstm_2"), parallel_layer(ff=None)]),
    # one head per key/value head, wide values, plain rotation of the whole head, two taps
    "wide": config_of([parallel_layer(heads=2, kv_heads=2, dim=72, vdim=136, rot={"base": 100.0, "dims": 72}, scale=0.11,
                                      right={"heads": 3, "kv_heads": 3, "dim": 104, "vdim": 16, "conv": 2}, ff=48),
                       memory_layer(heads=1, dim=136, vdim=40, gate_cap=20.0, kind="mlstm_2")], width=64, vocab=77, eps=1e-3,
                      side=8),
    # sizes that are no multiples of eight; eight query heads on one key/value head; five taps
    "odd": config_of([parallel_layer(heads=8, kv_heads=1, dim=18, vdim=10, rot={"base": 1e6, "dims": 4}, scale=0.5,
                                     right={"heads": 6, "kv_heads": 1, "dim": 10, "vdim": 33, "conv": 5}, ff=31),
                      memory_layer(heads=5, dim=7, vdim=9, gate_cap=1.0, ff=17)], width=50, vocab=61, side=3),
    # value heads wider than one cluster of thread blocks carries
    "tall": config_of([memory_layer(heads=1, dim=20, vdim=300), parallel_layer(right={"heads": 2, "kv_heads": 2, "dim": 12,
                                                                                      "vdim": 264, "conv": 4})], width=56, vocab=90),
    # a kernel's own tile sizes
    "square": config_of([memory_layer(heads=2, dim=64, vdim=128, gate_cap=15.0, ff=256),
                         parallel_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125,
                                        rot={"base": 10000.0, "dims": 32, "scaling": {"factor": 2.0, "original": 256,
                                                                                       "fast": 8.0, "slow": 1.0}},
                                        right={"heads": 2, "kv_heads": 1, "dim": 128, "vdim": 128, "conv": 4}, ff=192)],
                        width=128, vocab=320, side=32),
}

SANDWICHES = {
    # all sizes and constants different; keys shared across other masks and caps, a layer without feed-forward
    "kept": sandwich_config([
        window_layer(mlp=routed_mlp(5, 2, 48)), window_layer(softcap=3.0, size=14, keep_first=1, scale=0.7, mlp=dense_mlp(112)),
        window_layer(kv_from=0, size=5, keep_first=7, scale=0.3, softcap=8.0), window_layer(kv_from=1, size=None, mlp=routed_mlp(4, 1, 80))]),
    # one key/value head per head, wide values, every key visible, no cap, every expert chosen
    "plain": sandwich_config([
        window_layer(heads=2, kv_heads=2, dim=72, vdim=136, scale=0.11, softcap=None, size=None, mlp=routed_mlp(3, 3, 40)),
        window_layer(heads=3, kv_heads=1, dim=16, vdim=8, scale=0.25, softcap=30.0, size=40, keep_first=0, mlp=dense_mlp(48))],
        width=64, vocab=77, logit_scale=3.0),
    # sizes that are no multiples of eight, an odd width, a window of one token, a single expert
    "odd": sandwich_config([
        window_layer(heads=8, kv_heads=1, dim=18, vdim=10, scale=0.5, size=1, keep_first=2, mlp=routed_mlp(7, 2, 31)),
        window_layer(heads=4, kv_heads=2, dim=9, vdim=13, size=6, keep_first=1, mlp=routed_mlp(1, 1, 17)),
        window_layer(heads=4, kv_heads=2, dim=9, vdim=13, size=11, keep_first=4, kv_from=1, mlp=dense_mlp(29))], width=51, vocab=61),
    # the kernels' own tile sizes
    "square": sandwich_config([
        window_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, size=64, keep_first=64, softcap=20.0, mlp=routed_mlp(16, 4, 64)),
        window_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, size=128, keep_first=16, kv_from=0, mlp=dense_mlp(256))],
        width=128, vocab=320, logit_scale=1.0),
    # more query heads on a key/value head than an MMA tile has rows, many experts
    "many": sandwich_config([
        window_layer(heads=20, kv_heads=1, dim=32, vdim=48, size=33, keep_first=5, mlp=routed_mlp(40, 3, 24)),
        window_layer(heads=5, kv_heads=5, dim=128, vdim=128, scale=0.09, size=70, keep_first=2, mlp=routed_mlp(9, 2, 104))],
        width=96, vocab=130),
}


def settled_tokens(config, weights, length, seed=0, margin=0.08):
    """Random tokens none of whose choices of experts is a close call: tokens with one are drawn anew."""
    import oracle_mixers as plain

    rng = np.random.default_rng(seed)
    tokens = rng.integers(0, config["vocab"], size=length)
    for _ in range(1000):
        margins = []
        plain.forward_sandwich(config, weights, tokens, margins=margins)
        close = np.nonzero(np.min(margins, axis=0) < margin)[0] if margins else ()
        if not len(close):
            return tokens.tolist()
        tokens[close] = rng.integers(0, config["vocab"], size=len(close))
    raise AssertionError("no sequence of clear choices found")

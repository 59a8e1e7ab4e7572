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


def bf16_round(array):
    bits = np.ascontiguousarray(array, np.float32).view(np.uint32)
    return (((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def weights_of(config, seed=0):
    """fp32 arrays whose values are exact in bfloat16; every norm, gate and bias differs from the neutral value."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in mixer_tensors(parse_config(config)).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
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
            value = rng.standard_normal(shape) * 0.3
        elif leaf == "conv":
            value = rng.standard_normal(shape) * 0.5
        elif name in ("embed", "side.embed"):
            value = rng.standard_normal(shape)
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

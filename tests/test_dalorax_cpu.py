"""Host side of the Dalorax models: configuration, tensors, cache layout, records of a step, and the plain restatement
itself."""

import numpy as np
import pytest

import oracle_mixers as plain
from mixer_models import SANDWICHES, dense_mlp, routed_mlp, sandwich_config, settled_tokens, weights_of, window_layer


def test_registry_reads_every_size_from_the_config():
    from llmopt_b200 import model

    config = model.parse_config(SANDWICHES["kept"])
    assert (config.width, config.vocabulary, config.logit_scale, config.norm) == (104, 150, 0.7, "tanh")
    assert config.tied_head and config.sinusoid and config.token_side is None
    first, second, third, last = (layer.mixer for layer in config.layers)
    assert (first.heads, first.kv_heads, first.dim, first.vdim, first.scale, first.softcap) == (6, 3, 24, 40, 0.4, 5.0)
    assert (first.window.size, first.window.keep_first) == (9, 3) and first.gate and not first.prepared and first.kv_from is None
    assert third.kv_from == 0 and third.window.size == 5 and third.softcap == 8.0 and last.window is None and last.kv_from == 1
    experts = config.layers[0].feed_forward
    assert isinstance(experts, model.ExpertsSpec) and (experts.experts, experts.top, experts.width) == (5, 2, 48)
    assert config.layers[1].feed_forward == model.FeedForwardSpec(width=112, activation="silu", gated=True)
    assert config.layers[2].feed_forward is None
    assert model.parse_config(SANDWICHES["plain"]).layers[0].mixer.softcap is None
    assert model.kernel_family(config) == "attention"

    shapes = model.mixer_tensors(config)
    assert shapes["l0.norm1.alpha"] == () and shapes["l0.norm1b.b"] == (104,) and shapes["final.norm.alpha"] == ()
    assert shapes["l0.mix.g"] == (6 * 40, 104) and shapes["l0.mlp.router"] == (5, 104) and shapes["l0.mlp.e4.down"] == (104, 48)
    assert shapes["l1.mlp.gate"] == (112, 104) and "l2.norm2" not in shapes and "l2.mix.k" not in shapes
    assert "head" not in shapes and "l2.mix.q" in shapes and "l2.mix.v" not in shapes


@pytest.mark.parametrize("layers,message", [
    ([dict(window_layer(), type="other")], "unsupported layer type"),
    ([window_layer(mlp={"kind": "hashed"})], "feed-forward kind"),
    ([window_layer(heads=5, kv_heads=2)], "whole groups"),
    ([window_layer(size=0)], "sees at least"),
    ([window_layer(mlp=routed_mlp(4, 5, 8))], "at most all"),
    ([window_layer(kv_from=0)], "earlier attention layer"),
    ([window_layer(), window_layer(kv_from=0), window_layer(kv_from=1)], "has its own"),
    ([window_layer(), window_layer(kv_from=0, vdim=8)], "equal key and value heads")])
def test_registry_refuses_what_the_design_has_not(layers, message):
    from llmopt_b200 import model

    with pytest.raises(ValueError, match=message):
        model.parse_config(sandwich_config(layers))


class RecordingEngine:
    """The engine with a recorder in the place of the device."""

    def __new__(cls, config, **options):
        from unittest import mock

        from llmopt_b200 import mixer_engine, residual
        from llmopt_b200.model import parse_config, random_mixer_weights

        class FakeBuffer:
            def __init__(self, nbytes):
                self.nbytes = nbytes

        spec = parse_config(config)
        fake = mock.Mock()
        fake.create = lambda runtime, nbytes: FakeBuffer(nbytes)
        fake.of_array = lambda runtime, array: FakeBuffer(array.nbytes)
        with mock.patch.object(mixer_engine, "Buffer", fake), mock.patch.object(residual, "Buffer", fake):
            engine = mixer_engine.MixerEngine(None, spec, random_mixer_weights(spec), **options)
            engine.names = {}
            for sequences, tokens in ((1, 1), (3, 1), (1, 2), (1, 70), (1, 200)):
                plan = mixer_engine._Plan(engine, sequences, tokens)
                engine._record_layers(plan.step)
                engine.names[sequences, tokens] = [item.name for item in plan.items]
        return engine


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_records_of_a_step(dtype):
    """A dense layer is five launches, one without keys of its own too; few rows stream the experts' weights."""
    config = sandwich_config([window_layer(mlp=dense_mlp(64)), window_layer(kv_from=0, mlp=routed_mlp(6, 2, 32))])
    names = RecordingEngine(config, batch=3, capacity=256, dtype=dtype).names
    s = "bf16" if dtype == "bfloat16" else "f32"
    head = [f"llmopt_embedding_sinusoid_{s}", f"llmopt_dense_cached_{s}", f"llmopt_row_attention_{s}", f"llmopt_dense_residual_{s}",
            f"llmopt_dense_linear_{s}", f"llmopt_dense_residual_{s}",
            f"llmopt_dense_linear_{s}", f"llmopt_row_attention_{s}", f"llmopt_dense_residual_{s}", f"llmopt_dense_linear_{s}"]
    streamed = ["llmopt_route_step_f32", "llmopt_expert_step_bf16", "llmopt_expert_step_residual_bf16"]
    gathered = ["llmopt_route_rows_f32", "llmopt_route_plan", f"llmopt_gather_rows_{s}", f"llmopt_expert_rows_{s}",
                f"llmopt_expert_rows_{s}", f"llmopt_expert_combine_{s}"]
    for (sequences, tokens), recorded in names.items():
        assert recorded == head + (streamed if dtype == "bfloat16" and sequences * tokens <= 64 else gathered)


def test_cache_rows_of_layers_that_share_keys():
    engine = RecordingEngine(SANDWICHES["kept"], capacity=64)
    assert len(engine.layout.regions) == 2  # two of four layers have keys of their own
    regions = [layer.mixer.branches[0].region for layer in engine.layers]
    assert regions[2] is regions[0] and regions[3] is regions[1] and regions[0] is not regions[1]


def test_splits_follow_what_a_window_can_see():
    from llmopt_b200.mixers import Step

    engine = RecordingEngine(sandwich_config([window_layer(size=40, keep_first=6), window_layer(size=500, keep_first=0),
                                              window_layer(size=None)]), capacity=4096)
    step = Step(engine, 1, 1, None, None, None, None)
    with pytest.MonkeyPatch.context() as patch:
        patch.setattr(engine, "empty_bytes", lambda nbytes: nbytes)
        splits = [engine.attention_splits(step, layer.mixer)[0] for layer in engine.config.layers]
    assert splits == [1, 8, 64]


def test_attention_family_has_no_recurrent_kernels():
    import subprocess

    from llmopt_b200 import _build

    path = _build.build(family="attention")
    assert _build.current("attention") and path.endswith("libllmopt_cuda_attention.so")
    assert set(_build.FAMILIES["attention"]) < set(_build.FAMILIES["mixers"])
    names = subprocess.run(["strings", path], capture_output=True, text=True).stdout
    if names:  # binutils may be absent
        assert "llmopt_expert_step_bf16" in names and "llmopt_delta_scan_f32" not in names


# ---- the plain restatement itself ----------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(SANDWICHES))
def test_plain_restatement_is_causal_and_uses_every_tensor(name):
    config = SANDWICHES[name]
    weights = weights_of(config)
    tokens = settled_tokens(config, weights, 24, seed=1)
    base = plain.forward(config, weights, tokens)
    changed = list(tokens)
    changed[15] = (changed[15] + 1) % config["vocab"]
    other = plain.forward(config, weights, changed)
    assert np.allclose(base[:15], other[:15], rtol=0, atol=1e-9) and not np.allclose(base[15:], other[15:])
    idle = 0
    for tensor in weights:
        moved = dict(weights)
        moved[tensor] = weights[tensor] * 1.5 + 0.25
        moves = np.max(np.abs(plain.forward(config, moved, tokens) - base)) > 1e-6
        idle += not moves
        assert moves or ".mlp.e" in tensor, tensor
    # a few experts of many may have no token
    assert idle <= 0.3 * sum(".mlp.e" in tensor for tensor in weights)


def test_plain_windows_and_kept_tokens():
    places = np.arange(12)
    seen = plain.visible_keys(places, places, {"size": 3, "keep_first": 2})
    assert np.nonzero(seen[7])[0].tolist() == [0, 1, 5, 6, 7] and np.nonzero(seen[1])[0].tolist() == [0, 1]
    assert np.nonzero(seen[4])[0].tolist() == [0, 1, 2, 3, 4] and np.nonzero(seen[5])[0].tolist() == [0, 1, 3, 4, 5]
    assert np.array_equal(plain.visible_keys(places, places, None), np.tril(np.ones((12, 12), bool)))
    # portions of the queries see what they see in the whole
    assert np.array_equal(plain.visible_keys(places[5:9], places, {"size": 3, "keep_first": 2}), seen[5:9])


def test_plain_attention_by_hand():
    """Two keys, two values: the capped scores' softmax."""
    q, k, v = np.array([[[2.0]], [[3.0]]]), np.array([[[1.0]], [[-1.0]]]), np.array([[[10.0]], [[20.0]]])
    seen = np.tril(np.ones((2, 2), bool))
    out = plain.masked_attention(q, k, v, seen, 0.5, 2.0)
    scores = 2.0 * np.tanh(np.array([1.5, -1.5]) / 2.0)
    weights = np.exp(scores) / np.exp(scores).sum()
    assert out[0, 0, 0] == 10.0 and abs(out[1, 0, 0] - weights @ [10.0, 20.0]) < 1e-12


def test_plain_experts_scale_the_input():
    rng = np.random.default_rng(0)
    h = rng.standard_normal((1, 6))
    weights = {"m.router": rng.standard_normal((3, 6))}
    for e in range(3):
        weights |= {f"m.e{e}.gate": rng.standard_normal((4, 6)), f"m.e{e}.up": rng.standard_normal((4, 6)),
                    f"m.e{e}.down": rng.standard_normal((6, 4))}
    out = plain.routed_experts(h, weights, "m", {"experts": 3, "top": 2})
    scores = 1.0 / (1.0 + np.exp(-(weights["m.router"] @ h[0])))
    want = np.zeros(6)
    for e in np.argsort(-scores)[:2]:
        x = scores[e] * h[0]
        gate = weights[f"m.e{e}.gate"] @ x
        want += weights[f"m.e{e}.down"] @ (gate / (1.0 + np.exp(-gate)) * (weights[f"m.e{e}.up"] @ x))
    assert np.allclose(out[0], want)
    assert plain.chosen_experts(np.array([[1.0, 2.0, 2.0, 0.0]]), 3).tolist() == [[1, 2, 0]]


def test_plain_sinusoids():
    table = plain.sinusoids([0, 1, 1000], 5)
    assert table[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0]
    assert np.allclose(table[2], [np.sin(1000.0), np.cos(1000.0), np.sin(1000.0 * 10000 ** -0.4), np.cos(1000.0 * 10000 ** -0.4),
                                  np.sin(1000.0 * 10000 ** -0.8)])

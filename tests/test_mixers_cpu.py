"""Host side of the sequence-mixer models: configuration, checkpoint reader, rotary table, cache rows and the
owner of slots and state rows, the library of one kernel family."""

import json
import struct

import numpy as np
import pytest

import oracle_mixers as plain
from mixer_models import MODELS, config_of, memory_layer, parallel_layer, weights_of


def test_registry_reads_every_size_from_the_config():
    from llmopt_b200 import model

    config = model.parse_config(MODELS["mixed"])
    assert config.width == 104 and config.vocabulary == 150 and config.norm_offset == 1.0
    assert [type(layer.mixer).__name__ for layer in config.layers] == [
        "MatrixMemorySpec", "ParallelSpec", "MatrixMemorySpec", "ParallelSpec"]
    assert config.layers[2].feed_forward is None and config.layers[0].feed_forward.width == 112
    left, right = config.layers[1].mixer.left, config.layers[1].mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale) == (6, 3, 24, 40, 0.3)
    assert left.rotary.scaling.factor == 8.0 and left.bias and left.head_norm and left.sink
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.taps) == (4, 2, 36, 44, 3)
    shapes = model.mixer_tensors(config)
    assert shapes["l1.mix.right.v.conv"] == (4 * 44, 3) and shapes["l0.mix.norm"] == (72,)
    assert "l2.norm2" not in shapes and shapes["side.embed"] == (150, 4 * 24)
    with pytest.raises(ValueError, match="unsupported architecture"):
        model.parse_config({"architecture": "other"})
    with pytest.raises(ValueError, match="unsupported layer type"):
        model.parse_config(config_of([dict(memory_layer(), type="unknown")]))
    with pytest.raises(ValueError, match="feed-forward kind"):
        model.parse_config(config_of([dict(memory_layer(), mlp={"kind": "routed", "ff": 8})]))
    with pytest.raises(ValueError, match="whole groups"):
        model.parse_config(config_of([parallel_layer(heads=5, kv_heads=2)]))


def write_checkpoint(path, tensors):
    header, offset, payload = {}, 0, []
    for name, (dtype, array) in tensors.items():
        raw = array.tobytes()
        header[name] = {"dtype": dtype, "shape": list(array.shape), "data_offsets": [offset, offset + len(raw)]}
        payload.append(raw)
        offset += len(raw)
    text = json.dumps(header).encode()
    path.write_bytes(struct.pack("<Q", len(text)) + text + b"".join(payload))


def test_safetensors_reader(tmp_path):
    from llmopt_b200.safetensors_archive import Archive, as_bfloat16_bits, as_float32
    from llmopt_b200.weight_archive import ArchiveError

    values = np.array([[1.0, -2.5, 3.25], [0.0, 1e-3, 7.0]], np.float32)
    path = tmp_path / "model.safetensors"
    write_checkpoint(path, {"a": ("BF16", as_bfloat16_bits(values)), "b": ("I32", np.arange(5, dtype=np.int32)),
                            "c": ("F32", values)})
    archive = Archive(str(path))
    assert sorted(archive) == ["a", "b", "c"] and archive.find("a").shape == (2, 3) and "d" not in archive
    assert np.array_equal(as_float32(archive["a"])[0], values[0]) and np.array_equal(archive["b"], np.arange(5))
    assert np.array_equal(archive["c"], values) and archive.read("b") == np.arange(5, dtype=np.int32).tobytes()
    with pytest.raises(KeyError):
        archive["d"]
    # round to nearest even
    assert as_bfloat16_bits(np.array([1.00390625, 1.01171875, 1.0039064], np.float32)).tolist() == [0x3F80, 0x3F82, 0x3F81]
    path.write_bytes(path.read_bytes()[:-4])
    with pytest.raises(ArchiveError, match="exceeds the file"):
        Archive(str(path))
    path.write_bytes(struct.pack("<Q", 1 << 40))
    with pytest.raises(ArchiveError, match="index exceeds"):
        Archive(str(path))


@pytest.mark.parametrize("rot", [
    {"base": 10000.0, "dims": 48}, {"base": 500.0, "dims": 2},
    {"base": 10000.0, "dims": 64, "scaling": {"factor": 16.0, "original": 1024, "fast": 32.0, "slow": 1.0}},
    {"base": 20.0, "dims": 8, "scaling": {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 3.9}},
    {"base": 1e6, "dims": 16, "scaling": {"factor": 2.0, "original": 8, "fast": 64.0, "slow": 0.01}}])
def test_rotary_table(rot):
    from llmopt_b200.bizodra import _rotary
    from llmopt_b200.quantize import rotary_pairs

    table = rotary_pairs(3000, _rotary(rot))
    assert table.shape == (3000, rot["dims"] // 2, 2) and table.dtype == np.float32
    x = np.zeros((3000, 1, rot["dims"] + 6))
    x[:, :, 0:rot["dims"]:2] = 1.0  # (1, 0) pairs become (cos, sin)
    turned = plain.rotate(x, np.arange(3000), rot)
    assert np.allclose(table[..., 0], turned[:, 0, 0:rot["dims"]:2], atol=1e-6)
    assert np.allclose(table[..., 1], turned[:, 0, 1:rot["dims"]:2], atol=1e-6)


def test_row_layout_and_state_sizes():
    from llmopt_b200.kv_cache import RowLayout, matrix_state_elements

    layout = RowLayout([(3, 24, 40), (1, 18, 10)])
    assert [(r.key_offset, r.value_offset) for r in layout.regions] == [(0, 72), (192, 216)]
    assert layout.token_elements == 232 and RowLayout([]).token_elements == 8
    assert matrix_state_elements(2, 10, 33, normalized=False) == 660
    assert matrix_state_elements(3, 10, 33, normalized=True) == 990 + 3 * 2 * 11
    assert matrix_state_elements(1, 9, 3, normalized=False) == 28  # 27 rounded up


def test_sequence_table_hands_out_rows_and_pages_again():
    from llmopt_b200.kv_cache import SequenceTable

    table = SequenceTable(rows=3, stride=20, slots=28, page=4)
    a, b = table.open(), table.open()
    assert table.reserve(a, 5) == range(0, 8) and table.reserve(b, 9) == range(0, 12)
    table.advance(a, 5), table.advance(b, 9)
    assert table.reserve(a, 3) == range(8, 8)          # still on its second page
    table.advance(a, 3)
    assert table.reserve(a, 1) == range(8, 12)
    table.advance(a, 1)
    used = lambda row: set(table.table[row, :table.lengths[row]].tolist())
    assert not used(a) & used(b) and max(used(a) | used(b)) < 28
    with pytest.raises(ValueError, match="no free pages"):
        table.reserve(a, 11)
    with pytest.raises(ValueError, match="outgrow"):
        table.reserve(b, 12)
    first = table.table[b, :4].tolist()
    table.close(b)
    with pytest.raises(ValueError, match="not open"):
        table.reserve(b, 1)
    c = table.open()
    assert c == b and table.lengths[c] == 0            # the row is used again, from nothing
    table.reserve(c, 4)
    assert table.table[c, :4].tolist() == first        # and so is the page
    table.open()
    with pytest.raises(ValueError, match="no sequence row"):
        table.open()
    # everything comes back
    for row in range(3):
        table.close(row)
    assert len(table._free_pages) == 7 and sorted(table._free_rows) == [0, 1, 2]


def test_family_library_has_only_its_kernels():
    import ctypes

    from llmopt_b200 import _build

    path = _build.build(family="mixers")
    assert _build.current("mixers") and path.endswith("libllmopt_cuda_mixers.so")
    library = ctypes.CDLL(path)
    assert hasattr(library, "llmopt_cuda_prebaked_create") and hasattr(library, "llmopt_cuda_sample_f32")
    assert not hasattr(library, "llmopt_cuda_attention_q8_paged_static")


def test_fp32_sampler_is_the_fp16_sampler():
    from llmopt_b200 import _build, cuda_native

    _build.build()
    rng = np.random.default_rng(0)
    for seed in range(1, 40):
        row = rng.standard_normal(300).astype(np.float16)
        options = dict(temperature=[0.0, 0.8, 1.3][seed % 3], top_k=[0, 5][seed % 2], top_p=[0.0, 0.7][seed % 2],
                       min_p=[0.0, 0.05][seed // 2 % 2], seed=seed)
        assert cuda_native.sample_f32(row.astype(np.float32), **options) == cuda_native.sample_f16(
            row.tobytes(), row.size, **options)


def test_plain_restatement_is_causal_and_uses_every_tensor():
    """The oracle itself: a later token changes no earlier row, and no tensor is without effect."""
    config = MODELS["odd"]
    weights = weights_of(config)
    tokens = np.random.default_rng(1).integers(0, config["vocab"], size=12)
    base = plain.forward(config, weights, tokens)
    changed = tokens.copy()
    changed[8] = (changed[8] + 1) % config["vocab"]
    other = plain.forward(config, weights, changed)
    assert np.array_equal(base[:8], other[:8]) and not np.allclose(base[8:], other[8:])
    for name in weights:
        moved = dict(weights)
        moved[name] = weights[name] * 1.5 + 0.25
        assert np.max(np.abs(plain.forward(config, moved, tokens) - base)) > 1e-6, name

"""Host side of the Dabevik design, no GPU: configuration and tensor reading, registry, trace bookkeeping,
and properties of the oracle itself."""
import io
import json
import os

import numpy as np
import pytest

import dabevik_oracle as o

LAYERS = [o.make_layer(), o.make_layer(heads=3, kv_heads=3, dim=10, vdim=14, size=5, keep_first=0, ff=None), o.make_layer(weights_of=0)]


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    cfg = o.make_config(layers=LAYERS)
    return o.save_model(str(tmp_path_factory.mktemp("m")), cfg, o.make_weights(cfg, 1)), cfg


def test_registry_finds_the_design(folder):
    from torchburn_b200 import models

    assert models.find_design({"architecture": "Dabevik"}).name == "dabevik"
    assert models.find_design({"model_type": "qwen2"}).name == "llama-int4"
    assert models.find_design({"architectures": ["LlamaForCausalLM"]}).name == "llama-int4"
    with pytest.raises(ValueError, match="no registered design"):
        models.find_design({"architecture": "other"})
    with pytest.raises(NotImplementedError, match="not in int3"):
        models.load_model(folder[0], "int3")


def test_layer_specs_follow_the_configuration(folder):
    from torchburn_b200 import dabevik

    s = dabevik.layer_specs(folder[1])
    assert [x.num_heads for x in s] == [4, 3, 4] and [x.ff for x in s] == [88, 0, 88]
    assert s[2].weights_of == 0 and s[0].weights_of is None
    assert (s[1].mask_window, s[1].mask_keep_first, s[0].value_dim) == (5, 0, 20)
    bad = o.make_config(layers=[dict(o.make_layer(), type="other")])
    with pytest.raises(NotImplementedError):
        dabevik.layer_specs(bad)


def test_checkpoint_reader(folder, tmp_path):
    from torchburn_b200 import checkpoint, dabevik

    t = checkpoint.read_model_tensors(folder[0])
    cfg, w = o.load_model(folder[0])
    assert set(t) == set(w)
    for name in w:
        got = (t.bf16(name, w[name].shape).astype(np.uint32) << 16).view(np.float32)
        assert np.array_equal(got.astype(np.float64), w[name]), name
    with pytest.raises(ValueError, match="shape"):
        t.bf16("embed", (1, 2))
    with pytest.raises(KeyError, match="missing"):
        t.bf16("nothing", (1,))
    names = dabevik.layer_tensors(t, 0, cfg["layers"][0], cfg["width"], cfg["canon"]["taps"])
    assert set(names) >= {"talk", "conv1", "conv2", "act"}
    names = dabevik.layer_tensors(t, 1, cfg["layers"][1], cfg["width"], cfg["canon"]["taps"])
    assert "up_w" not in names and "conv2" not in names
    bad = tmp_path / "x.safetensors"
    head = json.dumps({"a": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 8]}}).encode()
    bad.write_bytes(len(head).to_bytes(8, "little") + head + b"\0" * 4)   # truncated
    with pytest.raises(ValueError, match="bad offsets"):
        checkpoint.read_safetensors(str(bad))


def test_trace_gives_sequences_back_and_keeps_the_order_of_places(tmp_path):
    from torchburn_b200 import _lib, trace

    class Toy:
        max_batch, vocab_size = 2, 3

        def __init__(self):
            self.calls = []

        def extend(self, tokens, start, want, seq):
            self.calls.append((list(tokens), start, seq))
            return np.array([[seq, start + w, tokens[w]] for w in want], np.float32).reshape(len(want), 3)

        def reset_sequence(self, seq):
            self.calls.append(("end", seq))

    toy, said = Toy(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [9], "want": []}, {"id": "a", "tokens": [8], "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [1], "want": [0]}], "end": ["c", "b"]}]
    orig = _lib.lib
    _lib.lib = lambda: type("L", (), {"tb_device_fault_flag": staticmethod(lambda: 0)})
    try:
        trace.run(toy, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    finally:
        _lib.lib = orig
    assert said == ["done 0", "done 1", "done 2"]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [0, 2, 7, 0, 0, 5]
    assert np.fromfile(tmp_path / "1.f32", "<f4").tolist() == [0, 3, 8]
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [0, 0, 1]      # a's sequence, from position 0
    assert toy.calls[2] == ([8], 3, 0) and ("end", 1) in toy.calls


def test_trace_program_refuses_an_unserved_dtype(folder, tmp_path):
    from torchburn_b200 import trace

    assert trace.main(["--model", folder[0], "--dtype", "float8", "--out", str(tmp_path)]) == 3


def test_partial_library_builds_and_exports_the_abi():
    import ctypes

    from torchburn_b200 import _lib, build

    L = ctypes.CDLL(build.build(profile="dense"))
    assert all(hasattr(L, name) for name in _lib.SIGNATURES)
    assert set(build.sources("dense")) & set(build.INT4_SOURCES) == set()
    L.tb_gemv_w4a32_grouped.restype = ctypes.c_int32
    buf, wb = (ctypes.c_float * 64)(), (ctypes.c_uint8 * 128)()
    args = [ctypes.c_void_p(ctypes.addressof(b)) if b is not None else None for b in (buf, wb, buf, None, buf)]
    assert L.tb_gemv_w4a32_grouped(*args, ctypes.c_int64(4), ctypes.c_int64(64), ctypes.c_int32(32), None) == 9   # TB_ERR_UNSUPPORTED


def test_create_layered_validates_before_the_device():
    import torchburn_b200 as tb

    z = np.zeros((8, 8), np.uint16)
    kw = dict(hidden_size=8, vocab_size=8, norm_eps=1e-5, max_seq_len=8)
    with pytest.raises(ValueError, match="divisible by num_kv_heads"):
        tb.LayeredDecoder([tb.LayerSpec(3, 2, 4, 4, 1.0)], z, z, **kw)
    with pytest.raises(ValueError, match="non-positive"):
        tb.LayeredDecoder([tb.LayerSpec(2, 2, 4, 0, 1.0)], z, z, **kw)
    with pytest.raises(ValueError, match="uint16"):
        tb.LayeredDecoder([tb.LayerSpec(2, 2, 4, 4, 1.0)], z.astype(np.float32), z, **kw)
    with pytest.raises(ValueError, match="dtype"):
        tb.LayeredDecoder([tb.LayerSpec(2, 2, 4, 4, 1.0)], z, z, dtype="float16", **kw)


# ------------------------------------------------------------------ the oracle
def test_oracle_visibility():
    m = o.visible(12, 4, 2)
    assert m[9].nonzero()[0].tolist() == [0, 1, 6, 7, 8, 9]
    assert m[3].nonzero()[0].tolist() == [0, 1, 2, 3]
    assert o.visible(6, 1, 0).tolist() == np.eye(6, dtype=bool).tolist()


def test_oracle_convolution_is_causal():
    h = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    out = o.causal_conv(h, w)
    assert out[0].tolist() == [0.0, 1.0]
    assert out[3].tolist() == [100 * 6 + 10 * 4 + 1 * 2, 7.0]


def test_oracle_polynorm():
    z = np.array([[1.0, -2.0, 3.0]])
    got = o.polynorm(z, (2.0, 3.0, 5.0, 7.0), 0.0)
    want = 2 * z / np.sqrt(14 / 3) + 3 * z ** 2 / np.sqrt((1 + 16 + 81) / 3) + 5 * z ** 3 / np.sqrt((1 + 64 + 729) / 3) + 7
    assert np.allclose(got, want)


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = o.make_config(layers=LAYERS)
    w = o.make_weights(cfg, 3)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 30)
    assert np.allclose(o.forward(cfg, w, toks)[:17], o.forward(cfg, w, toks[:17]), atol=1e-9)

"""Host side of the Sukalorn design, no GPU: configuration and tensor reading, registry, refused combinations, and
properties of the oracle itself."""
import numpy as np
import pytest

import sukalorn_oracle as o

LAYERS = [o.latent_layer(), o.attention_layer(), o.attention_layer(heads=2, vdim=20, size=5, ff=None), o.attention_layer(v_mix=False, vdim=6)]


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    cfg = o.make_config(layers=LAYERS)
    return o.save_model(str(tmp_path_factory.mktemp("m")), cfg, o.make_weights(cfg, 1)), cfg


def test_registry_finds_the_design(folder):
    from torchburn_b200 import models

    assert models.find_design({"architecture": "Sukalorn"}).name == "sukalorn"
    assert "sukalorn" in models.designs()
    with pytest.raises(NotImplementedError, match="not in float16"):
        models.load_model(folder[0], "float16")


def test_layer_specs_follow_the_configuration(folder):
    from torchburn_b200 import sukalorn

    s = sukalorn.layer_specs(folder[1])
    assert [x.kv_rank for x in s] == [40, 0, 0, 0] and [x.ff for x in s] == [88, 88, 0, 88]
    assert [x.mask_chunk for x in s] == [0, 9, 5, 9] and [x.value_mix for x in s] == [False, True, True, False]
    assert (s[0].head_dim, s[0].rot_dim, s[0].rot_dims, s[0].rot_base, s[0].q_rank) == (20, 12, 12, 300.0, 52)
    assert (s[1].score_softcap, s[1].distance_bias, s[1].qk_unit_norm, s[1].num_kv_heads) == (7.0, 8.0, True, 2)
    with pytest.raises(NotImplementedError, match="mixer type"):
        sukalorn.layer_specs(o.make_config(layers=[dict(o.attention_layer(), type="other")]))
    with pytest.raises(NotImplementedError, match="feed-forward kind"):
        sukalorn.layer_specs(o.make_config(layers=[dict(o.attention_layer(), mlp={"kind": "other", "ff": 3})]))


def test_tensors_are_checked_against_the_configuration(folder):
    from torchburn_b200 import checkpoint, sukalorn

    t = checkpoint.read_model_tensors(folder[0])
    cfg = folder[1]
    assert set(sukalorn.layer_tensors(t, 0, cfg["layers"][0], cfg["width"])) >= {"dq_w", "dq_norm", "uq_w", "dkv_w", "dkv_norm", "uk_w", "uv_w"}
    names = sukalorn.layer_tensors(t, 2, cfg["layers"][2], cfg["width"])
    assert "up_w" not in names and names["vmix"].size == 1 and names["gate_w"].shape == (2, cfg["width"])
    assert "vmix" not in sukalorn.layer_tensors(t, 3, cfg["layers"][3], cfg["width"])
    bad = dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], kv_rank=41))
    with pytest.raises(ValueError, match="shape"):
        sukalorn.layer_tensors(t, 0, bad, cfg["width"])


def test_create_refuses_bad_sizes_before_the_device():
    import torchburn_b200 as tb

    z = np.zeros((8, 8), np.uint16)
    kw = dict(hidden_size=8, vocab_size=8, norm_eps=1e-5, max_seq_len=8)
    latent = dict(q_rank=4, kv_rank=4, rot_dim=4, rot_dims=4, rot_base=10.0)
    for change, message in ((dict(num_kv_heads=2), "one key/value head"), (dict(rot_dims=3), "rotation"), (dict(rot_dims=6), "rotation"),
                            (dict(q_rank=0), "latent"), (dict(rot_base=0.0), "rotation")):
        args = dict(dict(num_heads=2, num_kv_heads=1, head_dim=4, value_dim=4, score_scale=1.0, **latent), **change)
        with pytest.raises(ValueError, match=message):
            tb.LayeredDecoder([tb.LayerSpec(**args)], z, z, **kw)
    with pytest.raises(ValueError, match="negative"):
        tb.LayeredDecoder([tb.LayerSpec(2, 2, 4, 4, 1.0, mask_chunk=-1)], z, z, **kw)
    with pytest.raises(ValueError, match="activation"):
        tb.LayeredDecoder([tb.LayerSpec(2, 2, 4, 4, 1.0, ff=8, activation="other")], z, z, **kw)


# ------------------------------------------------------------------ the oracle
def test_oracle_chunks():
    m = o.same_chunk(12, 5)
    assert m[4].nonzero()[0].tolist() == [0, 1, 2, 3, 4] and m[5].nonzero()[0].tolist() == [5] and m[11].nonzero()[0].tolist() == [10, 11]


def test_oracle_rotation():
    x = np.ones((3, 1, 6))
    y = o.rotate(x, 100.0, 4)
    assert np.allclose(y[0], x[0]) and np.allclose(y[:, :, 4:], 1.0)
    assert np.allclose(y[2, 0, :2], [np.cos(2) - np.sin(2), np.cos(2) + np.sin(2)])
    assert np.allclose(y[2, 0, 2:4], [np.cos(0.2) - np.sin(0.2), np.cos(0.2) + np.sin(0.2)])


def test_oracle_bias_and_cap():
    assert np.allclose(o.slopes(4), [0.25, 0.0625, 0.015625, 0.00390625])
    assert np.allclose(o.distance_bias(6, 2)[0, 5, 1], 4 * 2.0 ** -4)
    assert np.allclose(o.softcap(np.array([0.0, 1e9, -1e9]), 3.0), [0.0, 3.0, -3.0])


def test_oracle_prefix_does_not_depend_on_what_follows():
    cfg = o.make_config(layers=LAYERS)
    w = o.make_weights(cfg, 3)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 30)
    assert np.allclose(o.forward(cfg, w, toks)[:17], o.forward(cfg, w, toks[:17]), atol=1e-9)

"""The Sukalorn design on the GPU against the plain float64 oracle, at sizes of these tests' own, and the flash
attention kernels with the masks that other designs use."""
import numpy as np
import pytest

import dabevik_oracle as dab
import sukalorn_oracle as o

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ["float32", "bfloat16"]

MODELS = {
    # both mixers, grouped heads, value size other than key size, layers without feed-forward or without mixed values
    "mixed": o.make_config(vocab=150, width=72, layers=[
        o.latent_layer(3, 20, 12, 18, 40, 52, ff=88), o.attention_layer(6, 2, 24, 20, 9, ff=88), o.attention_layer(6, 2, 16, 20, 14, cap=3.0, ff=None),
        o.attention_layer(2, 2, 24, 36, 33, v_mix=False, ff=40), o.latent_layer(5, 16, 8, 24, 24, 30, base=40.0, ff=None),
        o.attention_layer(4, 2, 30, 20, 21, scale=0.4, ff=200)]),
    # one head, chunks of one position, odd sizes, only a part of the rotated dimensions turning
    "edges": o.make_config(vocab=70, width=132, eps=1e-3, layers=[
        o.attention_layer(1, 1, 10, 7, 1, ff=64), o.latent_layer(1, 9, 6, 5, 11, 7, rot_dims=2, ff=36), o.attention_layer(5, 1, 33, 7, 4, ff=36)]),
    # more (query, head) pairs than one block of rows takes, in decode steps too
    "many": o.make_config(vocab=110, width=96, layers=[
        o.latent_layer(20, 24, 16, 48, 200, 64, scale=0.2, ff=130), o.attention_layer(24, 1, 72, 56, 50, scale=0.3, ff=None),
        o.latent_layer(70, 8, 4, 8, 32, 40, ff=60)]),
    # several tiles of everything, latents wider than half a kernel's columns
    "wide": o.make_config(vocab=700, width=264, layers=[
        o.latent_layer(12, 64, 32, 64, 384, 200, scale=0.12, base=10000.0, ff=520), o.attention_layer(16, 4, 128, 96, 100, scale=0.15, cap=20.0, ff=136),
        o.attention_layer(8, 4, 160, 96, 70, scale=0.15, ff=None)]),
    # sizes that the tcgen05 kernel of portions takes, with the cap's small arguments and without
    "even": o.make_config(vocab=130, width=128, layers=[
        o.attention_layer(8, 2, 64, 64, 200, scale=0.1, cap=30.0, ff=256), o.latent_layer(6, 32, 16, 40, 136, 72, ff=None),
        o.attention_layer(6, 2, 48, 64, 77, scale=0.5, cap=5.0, ff=96), o.latent_layer(4, 128, 64, 128, 512, 96, scale=0.07, ff=80)]),
    # head sizes of exactly 64, 128 and 256, many heads over a wide latent, more heads than a block of the decode kernel takes
    "heads": o.make_config(vocab=100, width=160, layers=[
        o.attention_layer(4, 2, 128, 128, 90, scale=0.1, cap=25.0, ff=72), o.latent_layer(24, 32, 16, 32, 512, 60, scale=0.15, ff=None),
        o.attention_layer(2, 1, 256, 256, 64, scale=0.07, v_mix=False, ff=None), o.attention_layer(8, 1, 64, 64, 150, scale=0.2, v_mix=False, ff=96),
        o.latent_layer(36, 16, 16, 24, 96, 48, scale=0.2, ff=None)]),
    # latents and keys beyond the tensor-core kernels' tiles, and at the limit of their shared memory
    "large": o.make_config(vocab=60, width=64, layers=[
        o.latent_layer(3, 12, 20, 16, 720, 48, ff=48), o.attention_layer(2, 1, 240, 16, 60, scale=0.05, v_mix=False, ff=None),
        o.latent_layer(4, 224, 32, 16, 64, 40, scale=0.06, ff=None), o.attention_layer(2, 2, 500, 300, 70, scale=0.05, v_mix=False, ff=40)]),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(MODELS.items()):
        w = o.make_weights(cfg, 10 + i)
        out[name] = (o.save_model(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


def tokens_for(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def err(got, want):
    """Root mean square difference of the worst row, relative to the logits' spread."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / want.std())


def load(path, dtype, **kw):
    import torchburn_b200 as tb

    return tb.load_model(path, dtype, **kw)


def fault():
    import torchburn_b200 as tb

    return tb.lib().tb_device_fault_flag()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_decoding(models, name, dtype):
    path, cfg, w = models[name]
    toks = tokens_for(cfg, 150, 1)
    want = o.forward(cfg, w, toks)
    dec = load(path, dtype, prefill_rows=64, max_seq_len=160)
    places = list(range(len(toks)))
    assert err(dec.extend(toks, 0, places), want) < TOL[dtype]
    for cuts in ([2] * 20, [3, 17, 2, 33, 5, 64, 2], [1, 2, 1, 100], [140], []):      # portions, then one by one
        dec.reset_sequence(0)
        rows, at = [], 0
        for c in cuts:
            rows.append(dec.extend(toks[at:at + c], at, list(range(c))))
            at += c
        while at < len(toks):
            rows.append(dec.step(toks[at], at)[None])
            at += 1
        assert err(np.concatenate(rows), want) < TOL[dtype], cuts
    dec.reset_sequence(0)
    order = [40, 3, 149, 7]
    assert err(dec.extend(toks, 0, order), want[order]) < TOL[dtype]
    assert err(dec.get_logits()[None], want[-1:]) < TOL[dtype]
    assert fault() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt_in_one_step(models, dtype):
    """Portions of several hundred rows, and a long cache behind short ones."""
    for name in ("mixed", "wide", "even"):
        path, cfg, w = models[name]
        toks = tokens_for(cfg, 430, 7)
        want = o.forward(cfg, w, toks)
        dec = load(path, dtype, prefill_rows=512, max_seq_len=3000)
        places = list(range(len(toks)))
        assert err(dec.extend(toks, 0, places), want) < TOL[dtype]
        dec.extend(toks[:421], 0)
        assert err(dec.extend(toks[421:], 421, list(range(9))), want[421:]) < TOL[dtype]
        dec.reset_sequence(0)
        dec.extend(toks[:420], 0)
        assert err(np.stack([dec.step(toks[p], p) for p in range(420, 430)]), want[420:]) < TOL[dtype]


def test_long_prompts_wrap_every_ring(models):
    """Portions of 64 positions and of odd sizes in front of rings that hold a chunk and 128 positions."""
    path, cfg, w = models["even"]
    toks = tokens_for(cfg, 1000, 17)
    want = o.forward(cfg, w, toks)
    dec = load(path, "bfloat16", prefill_rows=64, max_seq_len=1024)
    for cuts in ([1000], [100, 63, 65, 200, 129, 333, 110], [17, 400, 31, 552]):
        dec.reset_sequence(0)
        rows, at = [], 0
        for c in cuts:
            rows.append(dec.extend(toks[at:at + c], at, list(range(c))))
            at += c
        assert err(np.concatenate(rows), want) < TOL["bfloat16"], cuts
    assert fault() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "many"])
def test_residual_stream_after_every_layer(models, name, dtype):
    path, cfg, w = models[name]
    toks, layers = tokens_for(cfg, 21, 2), []
    o.forward(cfg, w, toks, layers)
    dec = load(path, dtype, debug=True)
    dec.extend(toks, 0, [])
    for i, want in enumerate(layers):
        got = dec.debug_stage(f"layer{i}").reshape(want.shape)
        assert np.abs(got - want).max() / np.abs(want).max() < TOL[dtype], i


def neutral(cfg, seed):
    """Weights whose values switch off what a value can: equal gates, no mixing, norms of weight one, no rotated part."""
    w = o.make_weights(cfg, seed)
    for name in w:
        if name.endswith((".g", "vmix", "embed.norm", "norm1", "norm2", "final.norm")):
            w[name] = np.zeros_like(w[name])
        elif name.endswith(("dq.norm", "dkv.norm")):
            w[name] = np.ones_like(w[name])
    for i, spec in enumerate(cfg["layers"]):
        m = spec["mixer"]
        if spec["type"] == "latent_attention":
            w[f"l{i}.mix.dkv"][m["kv_rank"]:] = 0
    return w


MECHANISMS = ["nothing", "softcap", "chunk", "mix.g", "mix.vmix", "embed.norm", "norm1", "norm2", "final.norm", "dq.norm", "dkv.norm", "rotation"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mechanism", MECHANISMS)
def test_each_mechanism_alone(tmp_path, mechanism, dtype):
    cap, size = (1.0 if mechanism == "softcap" else 1e4), (6 if mechanism == "chunk" else 500)
    kind = [o.latent_layer(4, 20, 8, 12, 24, 28, ff=72)] if mechanism in ("dq.norm", "dkv.norm", "rotation") else \
        [o.attention_layer(4, 2, 20, 12, size, cap=cap, ff=72)] * (2 if mechanism == "mix.vmix" else 1)
    cfg = o.make_config(vocab=90, width=56, layers=kind)
    full, w = o.make_weights(cfg, 5), neutral(cfg, 5)
    toks = tokens_for(cfg, 60, 3)
    off = o.make_config(vocab=90, width=56, layers=[dict(x, mixer=dict(x["mixer"], **({"softcap": 1e4, "mask": {"size": 500}} if x["type"] == "attention" else {})))
                                                   for x in kind])
    base = o.forward(off, w, toks)
    for name in w:
        if name.endswith(mechanism) or (mechanism == "rotation" and name.endswith("dkv")):
            w[name] = full[name]
    if mechanism == "mix.vmix":
        w["l1.mix.vmix"] = np.float64(0.625)
    want = o.forward(cfg, w, toks)
    if mechanism != "nothing":
        assert err(want, base) > 4 * TOL["bfloat16"]      # the mechanism shows
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype)
    got = np.concatenate([dec.extend(toks[:37], 0, list(range(37)))] + [dec.step(t, 37 + i)[None] for i, t in enumerate(toks[37:])])
    assert err(got, want) < TOL[dtype]


def test_the_fixed_mechanisms_show(models, monkeypatch):
    """What no weight switches off makes a difference in the models of these tests: the oracle without it fails the bar."""
    _, cfg, w = models["mixed"]
    toks = tokens_for(cfg, 60, 3)
    want = o.forward(cfg, w, toks)
    for name, without in (("distance_bias", lambda n, heads: np.zeros((heads, n, n))), ("rotate", lambda x, base, dims: x),
                          ("rms", lambda x, eps: x / 2), ("relu2", lambda z: np.maximum(z, 0)), ("softcap", lambda s, cap: s),
                          ("sigmoid", lambda x: np.ones_like(x)), ("mix_values", lambda v, first, lam: v), ("same_chunk", lambda n, size: o.causal(n))):
        with monkeypatch.context() as c:
            c.setattr(o, name, without)
            assert err(o.forward(cfg, w, toks), want) > 2 * TOL["bfloat16"], name


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [7, 1, 33, 32, 64, 100])
def test_chunk_edges_by_influence(tmp_path, size, dtype):
    """One layer: the logits at i depend on the token at j exactly when both lie in one chunk."""
    cfg = o.make_config(vocab=50, width=48, layers=[o.attention_layer(4, 1, 16, 16, size, scale=0.1, ff=32)])
    dec = load(o.save_model(str(tmp_path), cfg, o.make_weights(cfg, 7)), dtype, prefill_rows=48)
    n = 230
    toks = tokens_for(cfg, n, 4)

    def run(tokens, split):
        dec.reset_sequence(0)
        rows = [dec.extend(tokens[:split], 0, list(range(split)))]
        rows += [dec.step(tokens[p], p)[None] for p in range(split, n)]
        return np.concatenate(rows)

    for split in (n, 60):
        base = run(toks, split)
        for i in (size, 2 * size - 1 if size > 1 else 5, 97, 200, n - 1):
            start = i // size * size
            for j in {0, start - 2, start - 1, start, start + 1, i - 1}:
                if not 0 <= j < i:
                    continue
                other = list(toks)
                other[j] = (other[j] + 17) % cfg["vocab"]
                moved = float(np.abs(run(other, split)[i] - base[i]).max())
                assert (moved > 1e-5) if j >= start else (moved == 0.0), (i, j, split, moved)


def needle_model(kind):
    """Token 300 + n is the key that token n asks for: the key side is the query side on permuted features, and the
    embedding of 300 + n is that of n under the permutation, so their score stands far above the hundreds of others.
    Returns the tokens with such pairs at the given places and the same without keys."""
    if kind == "latent":
        layer = o.latent_layer(4, 32, 8, 24, 48, 48, scale=0.6, base=1000.0, ff=64)
        pairs = [(0, 550), (1, 610), (63, 560), (64, 563), (101, 600), (119, 618), (579, 619), (255, 601), (256, 602)]
    else:
        layer = o.attention_layer(8, 4, 32, 24, 500, scale=0.6, cap=60.0, ff=64)   # one chunk ends at 500
        pairs = [(0, 450), (1, 499), (63, 460), (64, 463), (101, 498), (500, 618), (501, 619), (563, 600), (564, 601)]
    cfg = o.make_config(vocab=400, width=96, layers=[layer])
    w = o.make_weights(cfg, 11, sharp=1.0)
    rng = np.random.default_rng(5)
    perm = rng.permutation(cfg["width"])
    for n in range(len(pairs)):
        w["embed"][300 + n][perm] = w["embed"][n]
    w["embed.norm"][:] = 0
    w["l0.norm1"][:] = 0
    if kind == "latent":
        m = layer["mixer"]
        h, d, rd = m["heads"], m["dim"], m["rot_dim"]
        w["l0.mix.dkv"][:48] = 0
        w["l0.mix.dkv"][:48, perm] = w["l0.mix.dq"]
        w["l0.mix.dq.norm"][:] = 1
        w["l0.mix.dkv.norm"][:] = 1
        uq = w["l0.mix.uq"].reshape(h, d + rd, -1)
        uq[:, :d] = w["l0.mix.uk"].reshape(h, d, -1)
        uq[:, d:] *= 0.25
    else:
        q = w["l0.mix.q"].reshape(8, 32, -1)
        w["l0.mix.k"][:] = 0
        w["l0.mix.k"][:, perm] = q[::2].reshape(128, -1)
        q[1::2] = q[::2]                                    # both query heads of a key head
    toks = rng.integers(10, 290, 620).tolist()
    without = list(toks)
    for n, (j, i) in enumerate(pairs):
        toks[j], toks[i] = 300 + n, n
        without[i] = n
    return cfg, w, toks, without, pairs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["latent", "attention"])
def test_far_key_stands_out(tmp_path, kind, dtype):
    cfg, w, toks, without, pairs = needle_model(kind)
    want, lost = o.forward(cfg, w, toks), o.forward(cfg, w, without)
    assert all(err(lost[[i]], want[[i]]) > 4 * TOL["bfloat16"] for _, i in pairs)
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype, prefill_rows=128, max_seq_len=700)
    at = [i for _, i in pairs]
    assert err(dec.extend(toks, 0, at), want[at]) < TOL[dtype]
    cut = 540 if kind == "latent" else 440
    dec.reset_sequence(0)
    dec.extend(toks[:cut], 0)
    got = np.stack([dec.step(toks[p], p) for p in range(cut, 620)])
    assert err(got, want[cut:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_turn_by_their_angle(tmp_path, dtype):
    """A rotated part alone, thousands of positions out: a rounded angle or position would show."""
    cfg = o.make_config(vocab=64, width=48, layers=[o.latent_layer(2, 8, 16, 12, 16, 24, scale=1.0, base=50.0, ff=None)])
    w = o.make_weights(cfg, 3, sharp=1.5)
    w["l0.mix.uk"][:] = 0
    toks = tokens_for(cfg, 3000, 8)
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype, max_seq_len=3000)
    want = o.forward(cfg, w, toks)
    got = dec.extend(toks[:2990], 0, list(range(2900, 2990)))
    assert err(got, want[2900:2990]) < TOL[dtype]
    assert err(np.stack([dec.step(toks[p], p) for p in range(2990, 3000)]), want[2990:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "many", "even", "heads"])
def test_unequal_requests_in_one_decoder(models, name, dtype):
    """Several sequences, prompts of unequal length, stepped together; ended sequences are used again."""
    path, cfg, w = models[name]
    dec = load(path, dtype, max_batch=5, prefill_rows=32, max_seq_len=256)
    reqs = [tokens_for(cfg, n, 20 + n) for n in (40, 2, 77, 23, 61)]
    want = [o.forward(cfg, w, r) for r in reqs]
    tail = [6, 1, 12, 20, 3]
    for s, (r, k) in enumerate(zip(reqs, tail)):
        cut = len(r) - k
        assert err(dec.extend(r[:cut], 0, list(range(cut)), seq=s), want[s][:cut]) < TOL[dtype]
    for i in range(max(tail)):
        offs = [min(len(r) - k + i, len(r) - 1) for r, k in zip(reqs, tail)]      # finished rows repeat their last token
        got = dec.step_batch([r[p] for r, p in zip(reqs, offs)], offs)
        for s in range(5):
            assert err(got[s][None], want[s][[offs[s]]]) < TOL[dtype], (i, s)
    # sequence 2 and 0 are given to other requests, the others go on unharmed
    for s, n in ((2, 90), (0, 11)):
        dec.reset_sequence(s)
        r = tokens_for(cfg, n, 50 + n)
        assert err(dec.extend(r, 0, list(range(n)), seq=s), o.forward(cfg, w, r)) < TOL[dtype]
    more = reqs[3] + [5]
    assert err(dec.extend([5], len(reqs[3]), [0], seq=3), o.forward(cfg, w, more)[[-1]]) < TOL[dtype]


def test_rows_of_a_batch_do_not_disturb_each_other(models):
    path, cfg, w = models["wide"]
    one, many = load(path, "bfloat16"), load(path, "bfloat16", max_batch=7)
    r = tokens_for(cfg, 30, 9)
    a = np.stack([one.step(t, i) for i, t in enumerate(r)])
    others = [tokens_for(cfg, 30, 60 + s) for s in range(6)]
    b = np.stack([many.step_batch([x[i] for x in others[:3]] + [t] + [x[i] for x in others[3:]], [i] * 7)[3] for i, t in enumerate(r)])
    assert err(b, a.astype(np.float64)) < 4e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_wraps_every_ring(models, dtype):
    """More positions than the rings behind the chunks (chunk + 128) hold."""
    path, cfg, w = models["mixed"]
    dec = load(path, dtype, prefill_rows=16, max_seq_len=400)
    toks = tokens_for(cfg, 390, 6)
    want = o.forward(cfg, w, toks)
    dec.extend(toks[:9], 0)
    got = np.stack([dec.step(t, 9 + i) for i, t in enumerate(toks[9:])])
    assert err(got, want[9:]) < TOL[dtype]


def test_going_back(models):
    path, cfg, w = models["mixed"]
    dec = load(path, "float32", prefill_rows=32, max_seq_len=600)
    toks = tokens_for(cfg, 500, 12)
    dec.extend(toks, 0)
    other = toks[:420] + tokens_for(cfg, 30, 13)         # an earlier continuation point, other tokens
    assert err(dec.extend(other[420:], 420, list(range(30))), o.forward(cfg, w, other)[420:]) < TOL["float32"]
    with pytest.raises(ValueError, match="cannot go on"):
        dec.step(3, 460)
    with pytest.raises(ValueError, match="cannot go back"):
        dec.step(3, 100)
    assert err(dec.extend(toks[:5], 0, [4]), o.forward(cfg, w, toks[:5])[[4]]) < TOL["float32"]
    # dead rows: zero logits, nothing stored
    assert not dec.step(-1, 5).any() and not dec.step(3, 100000).any()
    assert err(dec.step(toks[5], 5)[None], o.forward(cfg, w, toks[:6])[[5]]) < TOL["float32"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,vdim", [(7, 3, 20), (1, 2, 20), (33, 0, 20), (64, 8, 24), (500, 4, 20), (33, 0, 24), (150, 0, 40), (500, 0, 24)])
def test_flash_attention_with_windows_and_kept_positions(size, keep, vdim, dtype):
    """Layers whose heads are not mixed run on the same kernels with a window and kept first positions."""
    import torchburn_b200 as tb

    cfg = dab.make_config(vocab=90, width=72, taps=3, layers=[dab.make_layer(6, 2, 24, vdim, size=size, keep_first=keep, ff=88)])
    w = dab.make_weights(cfg, 9)
    w["l0.mix.talk"] = np.eye(6)
    raw = {n: (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16) for n, a in w.items()}
    names = {"norm1": "norm1", "norm1_after": "norm1b", "conv1": "canon1", "q_w": "mix.q", "q_b": "mix.q.b", "k_w": "mix.k", "k_b": "mix.k.b",
             "v_w": "mix.v", "v_b": "mix.v.b", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm", "o_w": "mix.o", "o_b": "mix.o.b", "norm2": "norm2",
             "norm2_after": "norm2b", "conv2": "canon2", "up_w": "mlp.up", "down_w": "mlp.down", "act": "mlp.act"}
    spec = tb.LayerSpec(6, 2, 24, vdim, 0.21, size, keep, 88, None, {k: raw["l0." + v] for k, v in names.items()})
    dec = tb.LayeredDecoder([spec], raw["embed"], raw["final.norm"], raw["pos"], hidden_size=72, vocab_size=90, norm_eps=1e-5, max_seq_len=400,
                            embed_scale=3.0, conv_taps=3, dtype=dtype, prefill_rows=48)
    toks = tokens_for(cfg, 300, 5)
    want = dab.forward(cfg, w, toks)
    got = np.concatenate([dec.extend(toks[:240], 0, list(range(240)))] + [dec.step(t, 240 + i)[None] for i, t in enumerate(toks[240:])])
    assert err(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,chunk,cap", [(50, 0, 0.0), (0, 64, 0.0), (70, 90, 4.0)])
def test_latent_attention_with_the_other_masks_and_a_cap(tmp_path, monkeypatch, window, chunk, cap, dtype):
    """The mechanisms are not tied to the design: latents behind a window, in chunks, with capped scores."""
    import torchburn_b200 as tb
    from torchburn_b200 import checkpoint, sukalorn

    cfg = o.make_config(vocab=90, width=72, layers=[o.latent_layer(4, 64, 16, 32, 64, 48, scale=0.2, ff=88), o.latent_layer(4, 32, 16, 32, 128, 48, scale=0.2, ff=None)])
    w = o.make_weights(cfg, 9)
    n = 400
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    mask = (j <= i) & (i - j < (window or n)) & (i // (chunk or n) == j // (chunk or n))
    monkeypatch.setattr(o, "causal", lambda m: mask[:m, :m])
    if cap:
        plain = o.softmax
        monkeypatch.setattr(o, "softmax", lambda s, m: plain(o.softcap(s, cap), m))
    path = o.save_model(str(tmp_path), cfg, w)
    t, specs = checkpoint.read_model_tensors(path), sukalorn.layer_specs(cfg)
    for k, s in enumerate(specs):
        s.tensors = sukalorn.layer_tensors(t, k, cfg["layers"][k], cfg["width"])
        s.mask_window, s.mask_chunk, s.score_softcap = window, chunk, cap
    dec = tb.LayeredDecoder(specs, t["embed"], t["final.norm"], embed_norm=t["embed.norm"], head=t["head"], hidden_size=72, vocab_size=90,
                            norm_eps=1e-5, norm_offset=1.0, max_seq_len=n, dtype=dtype, prefill_rows=96)
    toks = tokens_for(cfg, n, 5)
    want = o.forward(cfg, w, toks)
    got = np.concatenate([dec.extend(toks[:300], 0, list(range(300)))] + [dec.step(x, 300 + k)[None] for k, x in enumerate(toks[300:])])
    assert err(got, want) < TOL[dtype]
    assert fault() == 0


def test_greedy_generation_and_schedulers(models):
    import random

    from torchburn_b200 import BatchedDecoder, SpeculativeDecoder

    path, cfg, w = models["mixed"]
    prompts = [tokens_for(cfg, n, 30 + n) for n in (5, 1, 19)]
    n_new = 12
    want = [o.greedy(cfg, w, p, n_new) for p in prompts]
    dec = load(path, "float32")
    for p, e in zip(prompts, want):
        dec.reset_kv_cache()
        if len(p) > 1:
            dec.prefill_tokens(p[:-1], 0)
        assert dec.generate_greedy(p[-1], len(p) - 1, n_new) == e
        dec.reset_kv_cache()
        if len(p) > 1:
            dec.prefill_tokens(p[:-1], 0)
        toks, end = dec.generate_loop(p[-1], len(p) - 1, n_new + 1, temperature=0.0)
        assert toks[1:] == e and end == len(p) + n_new
    batched = load(path, "float32", max_batch=3)
    assert BatchedDecoder(lambda: batched, 3, temperature=0.0).generate_batch(prompts, n_new) == want
    random.seed(0)
    spec = SpeculativeDecoder(load(path, "float32"), dec, K=3, temperature=0.0)
    assert spec.generate(prompts[2], n_new) == want[2] and spec.accepted > 0
    # a draft that is often wrong sends the target back
    draft = load(path, "bfloat16")
    real = draft.step
    draft.step = lambda t, p: real(t, p) if p % 2 else real(t, p)[::-1].copy()
    spec = SpeculativeDecoder(draft, dec, K=4, temperature=0.0)
    assert spec.generate(prompts[0], n_new) == want[0]


def test_command_line_and_trace_program(models, tmp_path):
    import json
    import os
    import subprocess
    import sys

    path, cfg, w = models["edges"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = tokens_for(cfg, 9, 2)
    r = subprocess.run([sys.executable, "-m", "torchburn_b200", "generate", "--model", path, "--dtype", "float32", "--max-new", "6",
                        "--tokens", ",".join(map(str, p))], cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()[-1].split(",")] == o.greedy(cfg, w, p, 6)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": p[:4], "want": [3, 1]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": p[4:], "want": [4]}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": p[2:5], "want": [2]}], "end": ["y"]}]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "16"],
                       input="".join(json.dumps(s) + "\n" for s in steps), cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and r.stdout.split() == ["done", "0", "done", "1", "done", "2"], r.stderr
    want = o.forward(cfg, w, p)
    got = np.concatenate([np.fromfile(tmp_path / f"{i}.f32", "<f4") for i in (0, 1)]).reshape(3, -1)
    assert err(got, want[[3, 1, 8]]) < TOL["float32"]
    assert err(np.fromfile(tmp_path / "2.f32", "<f4")[None], o.forward(cfg, w, p[2:5])[[2]]) < TOL["float32"]

"""The Dabevik design on the GPU against the plain float64 oracle, at sizes of these tests' own."""
import numpy as np
import pytest

import dabevik_oracle as o

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ["float32", "bfloat16"]

MODELS = {
    # grouped heads, value size other than key size, borrowed weights, a layer without feed-forward
    "mixed": o.make_config(vocab=150, width=72, taps=4, layers=[
        o.make_layer(6, 2, 24, 20, size=9, keep_first=3, ff=88), o.make_layer(3, 3, 10, 14, size=5, keep_first=0, ff=None),
        o.make_layer(6, 2, 24, 20, size=14, keep_first=1, ff=88, weights_of=0, scale=0.17), o.make_layer(4, 1, 48, 40, size=33, keep_first=6, ff=200)]),
    # no neighbours, the narrowest window, nothing kept; more kept than the window is wide
    "edges": o.make_config(vocab=70, width=132, taps=1, layers=[
        o.make_layer(2, 2, 16, 16, size=1, keep_first=0, ff=64), o.make_layer(5, 5, 8, 24, size=4, keep_first=17, ff=36)]),
    # one head, long taps
    "single": o.make_config(vocab=33, width=40, taps=7, scale=1.0, eps=1e-3, layers=[o.make_layer(1, 1, 64, 64, size=300, keep_first=2, ff=40)]),
    # several tiles of everything
    "wide": o.make_config(vocab=700, width=264, taps=2, layers=[
        o.make_layer(12, 4, 80, 64, size=70, keep_first=5, ff=520), o.make_layer(16, 16, 32, 48, size=50, keep_first=2, ff=136)]),
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
    dec = load(path, dtype, prefill_rows=64)
    places = list(range(len(toks)))
    assert err(dec.extend(toks, 0, places), want) < TOL[dtype]
    for cuts in ([2] * 20, [3, 17, 2, 33, 5, 64, 2], [1, 2, 1, 100], [140]):      # portions, then one by one
        dec.reset_sequence(0)
        rows, at = [], 0
        for c in cuts:
            rows.append(dec.extend(toks[at:at + c], at, list(range(c))))
            at += c
        while at < len(toks):
            rows.append(dec.step(toks[at], at)[None])
            at += 1
        assert err(np.concatenate(rows), want) < TOL[dtype], cuts
    # wanted places in any order; logits of the last position stay with the decoder
    dec.reset_sequence(0)
    order = [40, 3, 149, 7]
    assert err(dec.extend(toks, 0, order), want[order]) < TOL[dtype]
    assert err(dec.get_logits()[None], want[-1:]) < TOL[dtype]
    assert fault() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_after_every_layer(models, dtype):
    path, cfg, w = models["mixed"]
    toks, layers = tokens_for(cfg, 21, 2), []
    o.forward(cfg, w, toks, layers)
    dec = load(path, dtype, debug=True)
    dec.extend(toks, 0, [])
    for i, want in enumerate(layers):
        got = dec.debug_stage(f"layer{i}").reshape(want.shape)
        assert np.abs(got - want).max() / np.abs(want).max() < TOL[dtype], i


def neutral(cfg, seed):
    """Weights with every optional mechanism switched off by its values."""
    w = o.make_weights(cfg, seed)
    for name in w:
        if name.endswith(("canon1", "canon2", ".b")):
            w[name] = np.zeros_like(w[name])
        elif name.endswith("talk"):
            w[name] = np.eye(w[name].shape[0])
        elif name.endswith("act"):
            w[name] = np.array([1.0, 0, 0, 0])
        elif name == "pos":
            w[name] = np.zeros_like(w[name])
    return w


MECHANISMS = ["nothing", "canon1", "canon2", "talk", "act", "bias", "pos", "window"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mechanism", MECHANISMS)
def test_each_mechanism_alone(tmp_path, mechanism, dtype):
    size, keep = (6, 2) if mechanism == "window" else (400, 0)
    cfg = o.make_config(vocab=90, width=56, taps=3, layers=[o.make_layer(4, 2, 20, 12, size=size, keep_first=keep, ff=72)])
    full, w = o.make_weights(cfg, 5), neutral(cfg, 5)
    toks = tokens_for(cfg, 60, 3)
    base = o.forward(cfg, w, toks)
    for name in w:
        if name.endswith("." + mechanism) or name == mechanism or (mechanism == "bias" and name.endswith(".b")):
            w[name] = full[name]
    want = o.forward(cfg, w, toks)
    if mechanism not in ("nothing", "window"):
        assert err(want, base) > 5 * TOL["bfloat16"]      # the mechanism shows
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype)
    got = np.concatenate([dec.extend(toks[:37], 0, list(range(37)))] + [dec.step(t, 37 + i)[None] for i, t in enumerate(toks[37:])])
    assert err(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", [(7, 3), (1, 2), (33, 0), (32, 1), (64, 8)])
def test_window_edges_by_influence(tmp_path, size, keep, dtype):
    """One layer, no neighbours: the logits at i depend on the token at j exactly when i sees j."""
    cfg = o.make_config(vocab=50, width=48, taps=1, layers=[o.make_layer(2, 1, 16, 16, size=size, keep_first=keep, ff=32)])
    w = o.make_weights(cfg, 7, sharp=1.0)
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype, prefill_rows=48)
    n = 130
    toks = tokens_for(cfg, n, 4)

    def run(tokens, split):
        dec.reset_sequence(0)
        rows = [dec.extend(tokens[:split], 0, list(range(split)))]
        rows += [dec.step(tokens[p], p)[None] for p in range(split, n)]
        return np.concatenate(rows)

    for split in (n, 60):
        base = run(toks, split)
        for i in (size + keep + 3, 97, n - 1):
            for j in {0, keep - 1, keep, i - size - 1, i - size, i - size + 1, i - 1}:
                if not 0 <= j < i:
                    continue
                other = list(toks)
                other[j] = (other[j] + 17) % cfg["vocab"]
                moved = float(np.abs(run(other, split)[i] - base[i]).max())
                seen = bool(o.visible(n, size, keep)[i, j])
                assert (moved > 1e-4) if seen else (moved == 0.0), (i, j, split, moved)


def needle_model():
    """Token 300 + n is the key that token n asks for: the key projection is the query projection on permuted
    features, and the embedding of 300 + n is that of n under the permutation, so their score stands far above
    the hundreds of others.  Returns the tokens with such pairs at the given places and the same without keys."""
    cfg = o.make_config(vocab=400, width=96, taps=2, max_positions=800, layers=[
        o.make_layer(4, 4, 32, 24, size=500, keep_first=2, ff=None, scale=0.6), o.make_layer(4, 4, 32, 24, size=40, keep_first=4, ff=64, scale=0.6)])
    w = o.make_weights(cfg, 11, sharp=1.0)
    w["pos"][:] = 0
    rng = np.random.default_rng(5)
    perm = rng.permutation(cfg["width"])
    for n in range(8):
        w["embed"][300 + n][perm] = w["embed"][n]
    for l in (0, 1):
        p = f"l{l}."
        w[p + "mix.k"] = np.zeros_like(w[p + "mix.q"])
        w[p + "mix.k"][:, perm] = w[p + "mix.q"]
        w[p + "mix.q.b"] *= 0
        w[p + "mix.k.b"] *= 0
        w[p + "mix.q.norm"][:] = 1.0
        w[p + "mix.k.norm"][:] = 1.0
        w[p + "norm1"][:] = 1.0
        w[p + "canon1"] *= 0.25
    toks = rng.integers(10, 290, 620).tolist()
    pairs = [(1, 550), (0, 610), (63, 560), (64, 563), (101, 600), (119, 618), (579, 619)]   # kept, at the edge, far, near
    without = list(toks)
    for n, (j, i) in enumerate(pairs):
        toks[j], toks[i] = 300 + n, n
        without[i] = n
    return cfg, w, toks, without, pairs


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_stands_out(tmp_path, dtype):
    cfg, w, toks, without, pairs = needle_model()
    want, lost = o.forward(cfg, w, toks), o.forward(cfg, w, without)
    assert all(err(lost[[i]], want[[i]]) > 5 * TOL["bfloat16"] for _, i in pairs)
    dec = load(o.save_model(str(tmp_path), cfg, w), dtype, prefill_rows=128)
    at = [i for _, i in pairs]
    assert err(dec.extend(toks, 0, at), want[at]) < TOL[dtype]
    dec.reset_sequence(0)
    dec.extend(toks[:540], 0)
    got = np.stack([dec.step(toks[p], p) for p in range(540, 620)])
    assert err(got, want[540:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_decoder(models, dtype):
    """Several sequences, prompts of unequal length, stepped together; ended sequences are used again."""
    path, cfg, w = models["mixed"]
    dec = load(path, dtype, max_batch=5, prefill_rows=32)
    reqs = [tokens_for(cfg, n, 20 + n) for n in (40, 2, 77, 23, 61)]
    want = [o.forward(cfg, w, r) for r in reqs]
    tail = [6, 1, 12, 20, 3]
    for s, (r, k) in enumerate(zip(reqs, tail)):
        cut = len(r) - k
        assert err(dec.extend(r[:cut], 0, list(range(cut)), seq=s), want[s][:cut]) < TOL[dtype]
    for i in range(max(tail)):
        toks = [r[min(len(r) - k + i, len(r) - 1)] for r, k in zip(reqs, tail)]      # finished rows repeat their last token
        offs = [min(len(r) - k + i, len(r) - 1) for r, k in zip(reqs, tail)]
        got = dec.step_batch(toks, offs)
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
    assert err(b, a.astype(np.float64)) < 2e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_wraps_every_ring(models, dtype):
    """More positions than the cache rings (window + 128) and the convolution's history hold."""
    path, cfg, w = models["edges"]
    dec = load(path, dtype, prefill_rows=16)
    toks = tokens_for(cfg, 390, 6)
    want = o.forward(cfg, w, toks)
    dec.extend(toks[:9], 0)
    got = np.stack([dec.step(t, 9 + i) for i, t in enumerate(toks[9:])])
    assert err(got, want[9:]) < TOL[dtype]


def test_going_back(models):
    path, cfg, w = models["mixed"]
    dec = load(path, "float32", prefill_rows=32)
    toks = tokens_for(cfg, 300, 12)
    dec.extend(toks, 0)
    other = toks[:220] + tokens_for(cfg, 30, 13)         # an earlier continuation point, other tokens
    assert err(dec.extend(other[220:], 220, list(range(30))), o.forward(cfg, w, other)[220:]) < TOL["float32"]
    with pytest.raises(ValueError, match="cannot go on"):
        dec.step(3, 260)
    with pytest.raises(ValueError, match="cannot go back"):
        dec.step(3, 100)
    assert err(dec.extend(toks[:5], 0, [4]), o.forward(cfg, w, toks[:5])[[4]]) < TOL["float32"]
    # dead rows: zero logits, nothing stored
    assert not dec.step(-1, 5).any() and not dec.step(3, 100000).any()
    assert err(dec.step(toks[5], 5)[None], o.forward(cfg, w, toks[:6])[[5]]) < TOL["float32"]


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
    draft = load(models["mixed"][0], "bfloat16")
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
             {"step": 1, "entries": [{"id": "x", "tokens": p[4:], "want": [4]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "16"],
                       input="".join(json.dumps(s) + "\n" for s in steps), cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and r.stdout.split() == ["done", "0", "done", "1"], r.stderr
    want = o.forward(cfg, w, p)
    got = np.concatenate([np.fromfile(tmp_path / f"{i}.f32", "<f4") for i in (0, 1)]).reshape(3, -1)
    assert err(got, want[[3, 1, 8]]) < TOL["float32"]

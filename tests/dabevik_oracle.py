"""Plain float64 restatement of the Dabevik design, one function per mechanism.

Slow on purpose: whole sequences, no cache, no blocking; nothing is shared with the product package.
Weights are a dict name -> array with the checkpoint's tensor names, the configuration is the parsed
config.json.  ``make_config`` / ``make_weights`` build small random models for the tests.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def embed(cfg, w, tokens, start=0):
    tok = np.asarray(tokens)
    pos = np.arange(start, start + tok.size)
    return w["embed"][tok] * cfg["embedding"]["scale"] + w["pos"][pos]


def causal_conv(h, taps_w):
    """Per-channel causal convolution: the last tap multiplies the current position."""
    n, width = h.shape
    taps = taps_w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, width)), h], axis=0)
    out = np.zeros_like(h)
    for j in range(taps):
        out += taps_w[:, j] * padded[j:j + n]
    return out


def visible(n, size, keep_first):
    """mask[i, j]: position i sees position j."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def talk(t, p):
    """Post-softmax mixing of the heads' weights: p [H, i, j] -> sum_g t[h, g] p[g]."""
    return np.einsum("hg,gij->hij", t, p)


def project_qkv(h, w, pre, mixer, eps):
    heads, kv, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = h @ w[pre + "q"].T + w[pre + "q.b"]
    k = h @ w[pre + "k"].T + w[pre + "k.b"]
    v = h @ w[pre + "v"].T + w[pre + "v.b"]
    q = rms_norm(q, w[pre + "q.norm"], eps)   # over the whole projection, before the heads are split
    k = rms_norm(k, w[pre + "k.norm"], eps)
    return q.reshape(-1, heads, dim), k.reshape(-1, kv, dim), v.reshape(-1, kv, vdim)


def attention(h, w, pre, mixer, eps):
    heads, kv = mixer["heads"], mixer["kv_heads"]
    q, k, v = project_qkv(h, w, pre, mixer, eps)
    rep = heads // kv
    k, v = np.repeat(k, rep, axis=1), np.repeat(v, rep, axis=1)
    s = np.einsum("ihd,jhd->hij", q, k) * mixer["scale"]
    p = softmax(s, visible(h.shape[0], mixer["mask"]["size"], mixer["mask"]["keep_first"])[None])
    p = talk(w[pre + "talk"], p)
    o = np.einsum("hij,jhc->ihc", p, v).reshape(h.shape[0], -1)
    return o @ w[pre + "o"].T + w[pre + "o.b"]


def polynorm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def feed_forward(h, w, pre, eps):
    return polynorm(h @ w[pre + "up"].T, w[pre + "act"], eps) @ w[pre + "down"].T


def layer(cfg, w, i, x):
    spec = cfg["layers"][i]
    src = spec.get("weights_of")
    p = f"l{i if src is None else src}."
    eps = cfg["norm"]["eps"]
    h = rms_norm(x, w[p + "norm1"], eps)
    h = h + causal_conv(h, w[p + "canon1"])
    x = x + rms_norm(attention(h, w, p + "mix.", spec["mixer"], eps), w[p + "norm1b"], eps)
    if spec["mlp"] is not None:
        h = rms_norm(x, w[p + "norm2"], eps)
        h = h + causal_conv(h, w[p + "canon2"])
        x = x + rms_norm(feed_forward(h, w, p + "mlp.", eps), w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, layers_out=None):
    """Logits of every position, [n, vocab]."""
    x = embed(cfg, w, tokens)
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


# ------------------------------------------------------------------ small random models
def bf16(x):
    """Rounds to the nearest bfloat16 (ties to even), as float32."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def make_config(vocab=96, width=72, layers=None, taps=4, max_positions=400, eps=1e-5, scale=3.0):
    return {"architecture": "Dabevik", "vocab": vocab, "width": width, "max_positions": max_positions,
            "canon": {"taps": taps}, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


def make_layer(heads=4, kv_heads=2, dim=24, vdim=20, size=9, keep_first=3, scale=0.21, ff=88, weights_of=None):
    d = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                        "mask": {"size": size, "keep_first": keep_first}},
         "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def make_weights(cfg, seed=0, sharp=3.0):
    """Random weights, all bfloat16 values.  ``sharp`` scales the query/key norm weights so that the
    softmax is far from uniform and single keys matter."""
    rng = np.random.default_rng(seed)
    width = cfg["width"]
    out = {}

    def put(name, shape, std, mean=0.0):
        out[name] = bf16(mean + std * rng.standard_normal(shape)).astype(np.float64)

    put("embed", (cfg["vocab"], width), 0.4)
    put("pos", (cfg["max_positions"], width), 0.5)
    for i, spec in enumerate(cfg["layers"]):
        if spec.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", spec["mixer"]
        qn, kn, vn, on = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        for n in ["norm1", "norm1b"] + (["norm2", "norm2b"] if spec["mlp"] else []):
            put(p + n, (width,), 0.2, 1.0)
        put(p + "canon1", (width, cfg["canon"]["taps"]), 0.4)
        for n, rows in (("q", qn), ("k", kn), ("v", vn)):
            put(p + "mix." + n, (rows, width), 1.0 / math.sqrt(width))
            put(p + "mix." + n + ".b", (rows,), 0.3)
        put(p + "mix.q.norm", (qn,), 0.2, sharp)
        put(p + "mix.k.norm", (kn,), 0.2, 1.0)
        out[p + "mix.talk"] = bf16(np.eye(m["heads"]) + 0.5 * rng.standard_normal((m["heads"], m["heads"]))).astype(np.float64)
        put(p + "mix.o", (width, on), 1.0 / math.sqrt(on))
        put(p + "mix.o.b", (width,), 0.3)
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            put(p + "canon2", (width, cfg["canon"]["taps"]), 0.4)
            put(p + "mlp.up", (ff, width), 1.0 / math.sqrt(width))
            put(p + "mlp.down", (width, ff), 1.0 / math.sqrt(ff))
            put(p + "mlp.act", (4,), 0.5)
    put("final.norm", (width,), 0.2, 1.0)
    return out


def save_model(path, cfg, w):
    """Writes config.json and model.safetensors (bfloat16 tensors)."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, a in w.items():
        b = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)
    return path


def load_model(path):
    cfg = json.load(open(os.path.join(path, "config.json")))
    raw = open(os.path.join(path, "model.safetensors"), "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    w = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        u = np.frombuffer(raw[8 + n + lo:8 + n + hi], np.uint16).astype(np.uint32) << 16
        w[name] = u.view(np.float32).astype(np.float64).reshape(t["shape"])
    return cfg, w

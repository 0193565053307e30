"""Plain float64 restatement of the Sukalorn design, one function per mechanism.

Slow on purpose: whole sequences, no cache, no blocking, per-head keys and values written out; nothing is shared
with the product package.  Weights are a dict name -> array with the checkpoint's tensor names, the configuration
is the parsed config.json.  ``make_config`` / ``make_weights`` build small random models for the tests.
"""
from __future__ import annotations

import math

import numpy as np

from dabevik_oracle import bf16, load_model, save_model  # noqa: F401  (rounding and files, for the tests)


def rms(x, eps):
    """x over the root of its mean square (eps inside the root), last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """The model's norm: its weight is stored as the difference from one."""
    return rms(x, eps) * (1.0 + w)


def embed(cfg, w, tokens):
    return norm(w["embed"][np.asarray(tokens)], w["embed.norm"], cfg["norm"]["eps"])


def rotate(x, base, dims):
    """x [n, ..., d], row = position; dimensions 2i and 2i + 1 below ``dims`` turn by position * base^(-2i / dims)."""
    n = x.shape[0]
    a = np.arange(n)[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)[None, :]
    a = a.reshape((n,) + (1,) * (x.ndim - 2) + (dims // 2,))
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def causal(n):
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return j <= i


def same_chunk(n, size):
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return causal(n) & (i // size == j // size)


def softcap(s, cap):
    return cap * np.tanh(s / cap)


def slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def distance_bias(n, heads):
    """[H, i, j]: slope_h * (i - j)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return slopes(heads)[:, None, None] * (i - j)[None]


def softmax(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def attention(h, w, pre, m, eps, first_v=None):
    """Returns (output, values before mixing)."""
    n, heads, kv = h.shape[0], m["heads"], m["kv_heads"]
    q = rms((h @ w[pre + "q"].T).reshape(n, heads, m["dim"]), eps)
    k = rms((h @ w[pre + "k"].T).reshape(n, kv, m["dim"]), eps)
    own = (h @ w[pre + "v"].T).reshape(n, kv, m["vdim"])
    v = own if first_v is None else mix_values(own, first_v, float(w[pre + "vmix"]))
    k, v = np.repeat(k, heads // kv, axis=1), np.repeat(v, heads // kv, axis=1)
    s = softcap(np.einsum("ihd,jhd->hij", q, k) * m["scale"], m["softcap"]) - distance_bias(n, heads)
    p = softmax(s, same_chunk(n, m["mask"]["size"])[None])
    o = np.einsum("hij,jhc->ihc", p, v) * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(n, -1) @ w[pre + "o"].T, own


def latent_attention(h, w, pre, m, eps):
    n, heads, dim, rot, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    cq = rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (cq @ w[pre + "uq"].T).reshape(n, heads, dim + rot)
    d = h @ w[pre + "dkv"].T
    c = rms(d[:, :rank], eps) * w[pre + "dkv.norm"]
    k = (c @ w[pre + "uk"].T).reshape(n, heads, dim)
    v = (c @ w[pre + "uv"].T).reshape(n, heads, m["vdim"])
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    qr, kr = rotate(q[:, :, dim:], base, dims), rotate(d[:, rank:], base, dims)
    s = (np.einsum("ihd,jhd->hij", q[:, :, :dim], k) + np.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    o = np.einsum("hij,jhc->ihc", softmax(s, causal(n)[None]), v)
    return o.reshape(n, -1) @ w[pre + "o"].T


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def feed_forward(h, w, pre):
    return relu2(h @ w[pre + "up"].T) @ w[pre + "down"].T


def forward(cfg, w, tokens, layers_out=None):
    """Logits of every position, [n, vocab]."""
    eps = cfg["norm"]["eps"]
    x = embed(cfg, w, tokens)
    first_v = None
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if spec["type"] == "attention":
            y, own = attention(h, w, p + "mix.", m, eps, first_v if m.get("v_mix") else None)
            if m.get("v_mix") and first_v is None:
                first_v = own
        else:
            y = latent_attention(h, w, p + "mix.", m, eps)
        x = x + y
        if spec["mlp"] is not None:
            x = x + feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


# ------------------------------------------------------------------ small random models
def make_config(vocab=90, width=72, layers=None, eps=1e-5):
    return {"architecture": "Sukalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def _mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def attention_layer(heads=4, kv_heads=2, dim=24, vdim=20, size=9, scale=0.6, cap=7.0, v_mix=True, ff=88):
    return {"type": "attention", "mlp": _mlp(ff), "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "v_mix": v_mix, "mask": {"size": size}}}


def latent_layer(heads=3, dim=20, rot_dim=12, vdim=18, kv_rank=40, q_rank=52, scale=0.3, base=300.0, ff=88, rot_dims=None):
    return {"type": "latent_attention", "mlp": _mlp(ff), "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
        "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}}


def make_weights(cfg, seed=0, sharp=2.0):
    """Random weights, all bfloat16 values.  ``sharp`` scales the latent queries so that single keys matter."""
    rng = np.random.default_rng(seed)
    width = cfg["width"]
    out = {}

    def put(name, shape, std, mean=0.0):
        out[name] = bf16(np.asarray(mean + std * rng.standard_normal(shape), np.float32)).astype(np.float64).reshape(shape)

    put("embed", (cfg["vocab"], width), 0.7)
    put("embed.norm", (width,), 0.2)
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        x = p + "mix."
        put(p + "norm1", (width,), 0.2)
        if spec["type"] == "attention":
            h, kv, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            put(x + "q", (h * d, width), 1 / math.sqrt(width))
            put(x + "k", (kv * d, width), 1 / math.sqrt(width))
            put(x + "v", (kv * vd, width), 1 / math.sqrt(width))
            put(x + "vmix", (), 0.05, 0.4)
            put(x + "g", (h, width), 1.5 / math.sqrt(width))
            put(x + "o", (width, h * vd), 1 / math.sqrt(h * vd))
        else:
            h, d, rd, vd, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            put(x + "dq", (qr, width), 1 / math.sqrt(width))
            put(x + "dq.norm", (qr,), 0.2, 1.0)
            put(x + "uq", (h * (d + rd), qr), sharp / math.sqrt(qr))
            put(x + "dkv", (rank + rd, width), 1 / math.sqrt(width))
            put(x + "dkv.norm", (rank,), 0.2, 1.0)
            put(x + "uk", (h * d, rank), 1 / math.sqrt(rank))
            put(x + "uv", (h * vd, rank), 1 / math.sqrt(rank))
            put(x + "o", (width, h * vd), 1 / math.sqrt(h * vd))
        if spec["mlp"]:
            ff = spec["mlp"]["ff"]
            put(p + "norm2", (width,), 0.2)
            put(p + "mlp.up", (ff, width), 1 / math.sqrt(width))
            put(p + "mlp.down", (width, ff), 1 / math.sqrt(ff))
    put("final.norm", (width,), 0.2)
    put("head", (cfg["vocab"], width), 1 / math.sqrt(width))
    return out

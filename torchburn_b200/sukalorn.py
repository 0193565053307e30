"""The Sukalorn design: its config.json and tensor names on the layered decoder's mechanisms.

Two mixers in any order.  "attention": grouped heads without rotation, per-head query/key norms without a weight, a
soft cap on the scores and a distance bias, chunks of the sequence, values mixed with those of the first such
layer, a gate per head.  "latent_attention": queries and keys/values through normed latents, a rotated part of the
key that all heads share.  The feed-forward squares a relu; the embedding is normed; norm weights are stored around
zero; the output matrix is its own."""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional

from .checkpoint import Tensors
from .layered import LayeredDecoder, LayerSpec

DISTANCE_BIAS = 8.0            # head h of H: slope 2^(-8 (h + 1) / H)
NORM_OFFSET = 1.0
DEFAULT_POSITIONS = 4096       # the design has no longest sequence


def _attention(t: Tensors, p: str, m: Mapping[str, Any], width: int) -> Dict[str, Any]:
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    out = {
        "q_w": t.bf16(p + "q", (heads * dim, width)), "k_w": t.bf16(p + "k", (kv * dim, width)),
        "v_w": t.bf16(p + "v", (kv * vdim, width)), "gate_w": t.bf16(p + "g", (heads, width)),
        "o_w": t.bf16(p + "o", (width, heads * vdim)),
    }
    if m.get("v_mix"):
        out["vmix"] = t.bf16(p + "vmix", ())
    return out


def _latent(t: Tensors, p: str, m: Mapping[str, Any], width: int) -> Dict[str, Any]:
    heads, dim, rot, vdim, qr, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
    return {
        "dq_w": t.bf16(p + "dq", (qr, width)), "dq_norm": t.bf16(p + "dq.norm", (qr,)),
        "uq_w": t.bf16(p + "uq", (heads * (dim + rot), qr)), "dkv_w": t.bf16(p + "dkv", (kr + rot, width)),
        "dkv_norm": t.bf16(p + "dkv.norm", (kr,)), "uk_w": t.bf16(p + "uk", (heads * dim, kr)),
        "uv_w": t.bf16(p + "uv", (heads * vdim, kr)), "o_w": t.bf16(p + "o", (width, heads * vdim)),
    }


def layer_tensors(t: Tensors, i: int, spec: Mapping[str, Any], width: int) -> Dict[str, Any]:
    p = f"l{i}."
    out = (_latent if spec["type"] == "latent_attention" else _attention)(t, p + "mix.", spec["mixer"], width)
    out["norm1"] = t.bf16(p + "norm1", (width,))
    if spec.get("mlp") is not None:
        ff = spec["mlp"]["ff"]
        out.update({"norm2": t.bf16(p + "norm2", (width,)), "up_w": t.bf16(p + "mlp.up", (ff, width)),
                    "down_w": t.bf16(p + "mlp.down", (width, ff))})
    return out


def layer_specs(config: Mapping[str, Any]) -> List[LayerSpec]:
    """The layers' sizes and constants, without tensors."""
    out = []
    for i, spec in enumerate(config["layers"]):
        m, mlp = spec["mixer"], spec.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        common = dict(num_heads=m["heads"], head_dim=m["dim"], value_dim=m["vdim"], score_scale=m["scale"],
                      ff=mlp["ff"] if mlp is not None else 0, activation="relu2")
        if spec["type"] == "attention":
            out.append(LayerSpec(num_kv_heads=m["kv_heads"], mask_chunk=m["mask"]["size"], qk_unit_norm=True, score_softcap=m["softcap"],
                                 distance_bias=DISTANCE_BIAS, value_mix=bool(m.get("v_mix")), **common))
        elif spec["type"] == "latent_attention":
            out.append(LayerSpec(num_kv_heads=1, q_rank=m["q_rank"], kv_rank=m["kv_rank"], rot_dim=m["rot_dim"],
                                 rot_dims=m["rot"]["dims"], rot_base=m["rot"]["base"], **common))
        else:
            raise NotImplementedError(f"layer {i}: mixer type {spec['type']!r}")
    return out


def build(config: Mapping[str, Any], t: Tensors, dtype: str = "bfloat16", max_seq_len: Optional[int] = None, **kw) -> LayeredDecoder:
    width, vocab = config["width"], config["vocab"]
    specs = layer_specs(config)
    for i, (s, spec) in enumerate(zip(specs, config["layers"])):
        s.tensors = layer_tensors(t, i, spec, width)
    return LayeredDecoder(specs, t.bf16("embed", (vocab, width)), t.bf16("final.norm", (width,)), embed_norm=t.bf16("embed.norm", (width,)),
                          head=t.bf16("head", (vocab, width)), hidden_size=width, vocab_size=vocab, norm_eps=config["norm"]["eps"],
                          norm_offset=NORM_OFFSET, max_seq_len=max_seq_len or DEFAULT_POSITIONS, dtype=dtype, **kw)

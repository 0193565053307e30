"""The Dabevik design: its config.json and tensor names on the layered decoder's mechanisms.

Every sublayer reads h + conv(h) of its normed input and its output is normed before it is added; attention
has query/key norms over the whole projection, no rotation, a sliding window that keeps the first tokens, and
post-softmax mixing of the heads; the feed-forward's activation is PolyNorm; positions are a learned table;
the output matrix is the embedding.  Layers may borrow another layer's tensors (``weights_of``)."""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional

from .checkpoint import Tensors
from .layered import LayeredDecoder, LayerSpec


def layer_tensors(t: Tensors, i: int, spec: Mapping[str, Any], width: int, taps: int) -> Dict[str, Any]:
    m, mlp = spec["mixer"], spec.get("mlp")
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    p = f"l{i}."
    out = {
        "norm1": t.bf16(p + "norm1", (width,)), "norm1_after": t.bf16(p + "norm1b", (width,)),
        "conv1": t.bf16(p + "canon1", (width, taps)),
        "q_w": t.bf16(p + "mix.q", (heads * dim, width)), "q_b": t.bf16(p + "mix.q.b", (heads * dim,)),
        "k_w": t.bf16(p + "mix.k", (kv * dim, width)), "k_b": t.bf16(p + "mix.k.b", (kv * dim,)),
        "v_w": t.bf16(p + "mix.v", (kv * vdim, width)), "v_b": t.bf16(p + "mix.v.b", (kv * vdim,)),
        "q_norm": t.bf16(p + "mix.q.norm", (heads * dim,)), "k_norm": t.bf16(p + "mix.k.norm", (kv * dim,)),
        "talk": t.bf16(p + "mix.talk", (heads, heads)),
        "o_w": t.bf16(p + "mix.o", (width, heads * vdim)), "o_b": t.bf16(p + "mix.o.b", (width,)),
    }
    if mlp is not None:
        ff = mlp["ff"]
        out.update({
            "norm2": t.bf16(p + "norm2", (width,)), "norm2_after": t.bf16(p + "norm2b", (width,)),
            "conv2": t.bf16(p + "canon2", (width, taps)), "up_w": t.bf16(p + "mlp.up", (ff, width)),
            "down_w": t.bf16(p + "mlp.down", (width, ff)), "act": t.bf16(p + "mlp.act", (4,)),
        })
    return out


def layer_specs(config: Mapping[str, Any]) -> List[LayerSpec]:
    """The layers' sizes and constants, without tensors."""
    out = []
    for i, spec in enumerate(config["layers"]):
        if spec["type"] != "attention":
            raise NotImplementedError(f"layer {i}: mixer type {spec['type']!r}")
        m, mlp = spec["mixer"], spec.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        out.append(LayerSpec(
            num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], score_scale=m["scale"],
            mask_window=m["mask"]["size"], mask_keep_first=m["mask"]["keep_first"], ff=mlp["ff"] if mlp is not None else 0,
            weights_of=spec.get("weights_of")))
    return out


def build(config: Mapping[str, Any], t: Tensors, dtype: str = "bfloat16", max_seq_len: Optional[int] = None, **kw) -> LayeredDecoder:
    width, vocab, taps = config["width"], config["vocab"], config["canon"]["taps"]
    positions = config["max_positions"]
    seq = positions if max_seq_len is None else min(max_seq_len, positions)
    specs = layer_specs(config)
    for i, (s, spec) in enumerate(zip(specs, config["layers"])):
        if s.weights_of is None:
            s.tensors = layer_tensors(t, i, spec, width, taps)
    return LayeredDecoder(specs, t.bf16("embed", (vocab, width)), t.bf16("final.norm", (width,)),
                          t.bf16("pos", (positions, width))[:seq], hidden_size=width, vocab_size=vocab,
                          norm_eps=config["norm"]["eps"], max_seq_len=seq, embed_scale=config["embedding"]["scale"],
                          conv_taps=taps, dtype=dtype, **kw)

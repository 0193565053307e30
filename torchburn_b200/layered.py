"""Decoders described layer by layer (``tb_decoder_create_layered``): the mechanisms are the library's, a
design says which of them each layer has and with which constants."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Sequence

import numpy as np

from . import _lib
from ._lib import TB_DEVICE, TB_HOST, LAYERED_TENSORS, LayeredConfig, LayeredLayer, check, lib
from .decoder import DecoderHandle, _is_torch


@dataclass
class LayerSpec:
    """Sizes and constants of one layer, and its tensors by the names of ``tb_layered_layer`` (bfloat16: raw
    16-bit numpy arrays or torch tensors; a missing optional tensor leaves its mechanism out).  A layer with a
    ``kv_rank`` is latent attention (``num_kv_heads`` 1, ``head_dim`` its unrotated part)."""
    num_heads: int
    num_kv_heads: int
    head_dim: int
    value_dim: int
    score_scale: float
    mask_window: int = 0           # 0: no window
    mask_keep_first: int = 0
    ff: int = 0                    # 0: no feed-forward
    weights_of: Optional[int] = None
    tensors: Dict[str, Any] = field(default_factory=dict)
    activation: str = "polynorm"   # of the feed-forward: polynorm, relu2
    mask_chunk: int = 0            # 0: no chunks
    qk_unit_norm: bool = False     # per-head norm of queries and keys without a weight
    score_softcap: float = 0.0     # 0: none
    distance_bias: float = 0.0     # slope 2^(-distance_bias (h + 1) / heads); 0: none
    value_mix: bool = False
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_dims: int = 0
    rot_base: float = 0.0


_MLP = {"polynorm": _lib.TB_MLP_POLYNORM, "relu2": _lib.TB_MLP_RELU2}


class _Bf16Operands:
    """Keeps the arrays alive and yields raw pointers, all in one memory space."""

    def __init__(self):
        self.keep: List[Any] = []
        self.space: Optional[int] = None

    def ptr(self, a) -> Optional[int]:
        if a is None:
            return None
        if _is_torch(a):
            import torch

            t = a.detach().contiguous()
            if t.dtype != torch.bfloat16:
                raise ValueError(f"layered decoders take bfloat16 weights, got {t.dtype}")
            space, p = (TB_DEVICE if t.device.type == "cuda" else TB_HOST), t.data_ptr()
        else:
            t = np.ascontiguousarray(a)
            if t.dtype != np.uint16:
                raise ValueError(f"layered decoders take the raw bits of bfloat16 weights (uint16), got {t.dtype}")
            space, p = TB_HOST, t.ctypes.data
        if self.space is None:
            self.space = space
        elif self.space != space:
            raise ValueError("decoder weights must all live in the same memory space (all host or all CUDA)")
        self.keep.append(t)
        return p


class LayeredDecoder(DecoderHandle):
    """The package's decoder interface over a layered model.  ``dtype`` is "bfloat16" (products in bf16 with
    fp32 sums; residual, norms, scores and states fp32) or "float32" (everything)."""

    def __init__(self, layers: Sequence[LayerSpec], embed, final_norm, pos_table=None, *, hidden_size: int, vocab_size: int,
                 norm_eps: float, max_seq_len: int, embed_scale: float = 1.0, conv_taps: int = 0, dtype: str = "bfloat16",
                 max_batch: int = 1, prefill_rows: int = 0, debug: bool = False, pdl: bool = True, embed_norm=None, head=None,
                 norm_offset: float = 0.0):
        self._h = None
        if dtype not in _lib.TB_PRECISION:
            raise ValueError(f"dtype {dtype!r}: expected one of {sorted(_lib.TB_PRECISION)}")
        ops = _Bf16Operands()
        arr = (LayeredLayer * len(layers))()
        for dst, s in zip(arr, layers):
            unknown = set(s.tensors) - set(LAYERED_TENSORS)
            if unknown:
                raise ValueError(f"unknown layer tensors {sorted(unknown)}")
            if s.activation not in _MLP:
                raise ValueError(f"activation {s.activation!r}: expected one of {sorted(_MLP)}")
            dst.mixer = _lib.TB_MIXER_LATENT if s.kv_rank else _lib.TB_MIXER_ATTENTION
            dst.mlp = _MLP[s.activation] if s.ff else _lib.TB_MLP_NONE
            dst.weights_of = -1 if s.weights_of is None else s.weights_of
            dst.num_heads, dst.num_kv_heads, dst.head_dim, dst.value_dim = s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim
            dst.mask_window, dst.mask_keep_first, dst.score_scale, dst.ff = s.mask_window, s.mask_keep_first, s.score_scale, s.ff
            dst.mask_chunk, dst.qk_unit_norm, dst.score_softcap, dst.distance_bias = s.mask_chunk, s.qk_unit_norm, s.score_softcap, s.distance_bias
            dst.value_mix, dst.q_rank, dst.kv_rank = s.value_mix, s.q_rank, s.kv_rank
            dst.rot_dim, dst.rot_dims, dst.rot_base = s.rot_dim, s.rot_dims, s.rot_base
            for name, t in s.tensors.items():
                setattr(dst, name, ops.ptr(t))
        flags = (_lib.TB_DECODER_NO_GRAPH if debug else 0) | (0 if pdl else _lib.TB_DECODER_NO_PDL)
        self.cfg = LayeredConfig(vocab_size=vocab_size, hidden_size=hidden_size, num_layers=len(layers), conv_taps=conv_taps,
                                 norm_eps=norm_eps, embed_scale=embed_scale, max_seq_len=max_seq_len, max_batch=max_batch,
                                 prefill_rows=prefill_rows, precision=_lib.TB_PRECISION[dtype], flags=flags, norm_offset=norm_offset)
        tables = [ops.ptr(t) for t in (embed, embed_norm, pos_table, final_norm, head)]
        h = C.c_void_p()
        check(lib().tb_decoder_create_layered(C.byref(h), C.byref(self.cfg), C.cast(arr, C.c_void_p), *tables,
                                              ops.space if ops.space is not None else TB_HOST))
        self._adopt(h, vocab_size, max_batch, max_seq_len)

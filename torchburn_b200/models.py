"""The model registry: config.json -> the decoder that serves it.

``load_model(folder)`` reads the folder's config.json, finds the design that claims it and returns a decoder
(``DecoderHandle``) with the weights on the GPU."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, List, Mapping, Optional

from . import _lib, checkpoint
from .decoder import DecoderHandle


@dataclass(frozen=True)
class Design:
    name: str
    claims: Callable[[Mapping[str, Any]], bool]          # config -> is it this design?
    load: Callable[..., DecoderHandle]                   # (folder, config, dtype, max_seq_len, **options)
    dtypes: tuple                                        # what it can be served in
    profile: str = "full"                                # the library build it needs (build.py)


_DESIGNS: List[Design] = []


def register(design: Design) -> Design:
    _DESIGNS.append(design)
    return design


def designs() -> List[str]:
    return [d.name for d in _DESIGNS]


def find_design(config: Mapping[str, Any]) -> Design:
    for d in _DESIGNS:
        if d.claims(config):
            return d
    raise ValueError(f"no registered design for architecture {config.get('architecture') or config.get('architectures') or config.get('model_type')!r}")


def load_model(model_dir: str, dtype: Optional[str] = None, max_seq_len: Optional[int] = None, build: bool = False, **options) -> DecoderHandle:
    """``dtype`` None takes the design's first; ``build`` compiles the library the design needs if there is
    none; options (``max_batch``, ``prefill_rows``, ...) go to the design's decoder."""
    config = checkpoint.read_config(model_dir)
    d = find_design(config)
    dtype = dtype or d.dtypes[0]
    if dtype not in d.dtypes:
        raise NotImplementedError(f"{d.name} is served in {', '.join(d.dtypes)}, not in {dtype}")
    if build:
        from . import build as _build

        _lib.select(_build.ensure(d.profile))
    return d.load(model_dir, config, dtype, max_seq_len, **options)


# ------------------------------------------------------------------ the designs
def _load_dabevik(model_dir, config, dtype, max_seq_len, **options):
    from . import dabevik

    return dabevik.build(config, checkpoint.read_model_tensors(model_dir), dtype, max_seq_len, **options)


def _load_sukalorn(model_dir, config, dtype, max_seq_len, **options):
    from . import sukalorn

    return sukalorn.build(config, checkpoint.read_model_tensors(model_dir), dtype, max_seq_len, **options)


def _load_int4(model_dir, config, dtype, max_seq_len, group_size: int = 64, **options):
    """Llama / Qwen2 style checkpoints on the INT4 decoder: the folder's quantized cache if there is one, else
    its float tensors quantized on the GPU (python/torchburn/llm/loader.py:92-173, 376-537)."""
    import torch

    from . import loader

    layers, heads = config["num_hidden_layers"], config["num_attention_heads"]
    cache = loader.find_cache(model_dir, group_size)
    if cache:
        sd = loader.load_cache(cache)
    else:
        import safetensors.torch

        tensors = {}
        for path in checkpoint.weight_files(model_dir):
            tensors.update(safetensors.torch.load_file(path, device="cpu"))
        device = torch.device("cuda")

        def quantize(w):
            from .quantization import quantize_weight_int4_grouped

            return quantize_weight_int4_grouped(w.to(device), group_size=group_size)

        sd = loader.quantize_checkpoint(tensors, layers, group_size, config.get("tie_word_embeddings", False),
                                        config.get("attention_bias", config.get("model_type") == "qwen2"), quantize)
    qkv = sd["layers.0.self_attn.qkv_proj.scales"]
    hidden = config["hidden_size"]
    return loader.decoder_from_state_dict(
        sd, layers, hidden, config["intermediate_size"], heads, config.get("num_key_value_heads", heads),
        config.get("head_dim") or hidden // heads, hidden // qkv.shape[1], config.get("rms_norm_eps", 1e-6),
        max_seq_len or min(config.get("max_position_embeddings", 4096), 32768), config.get("rope_theta", 1e6), **options)


register(Design("dabevik", lambda c: c.get("architecture") == "Dabevik", _load_dabevik, ("bfloat16", "float32"), "dense"))
register(Design("sukalorn", lambda c: c.get("architecture") == "Sukalorn", _load_sukalorn, ("bfloat16", "float32"), "dense"))
register(Design("llama-int4", lambda c: c.get("model_type") in ("llama", "qwen2") or bool(
    {"LlamaForCausalLM", "Qwen2ForCausalLM"} & set(c.get("architectures") or ())), _load_int4, ("int4",)))

"""Model families by ``config.json``: which class runs a model folder, what it keeps between steps, and how its weights
come in.

``architecture`` (or the first of HF's ``architectures``) names the family.  A family is a ``ModelFamily``: parse the
configuration, build the model (from the folder's safetensors files, or random where a family has no checkpoint
reader), make its cache for a number of pages and state slots, and say what a page and a slot cost."""

from __future__ import annotations

import dataclasses
import json
import os
import types
from typing import Any

import torch

from .hybrid_config import HybridArgs


class ModelFamily:
    name = ""
    dtypes: tuple[torch.dtype, ...] = (torch.bfloat16,)
    component: str | None = None  # part of the kernel library that is enough for it (metal/build.py); None: all of it

    def parse(self, config: dict) -> Any:
        raise NotImplementedError

    def load(self, args: Any, folder: str | None, dtype: torch.dtype, device, seed: int = 0) -> Any:
        raise NotImplementedError

    def make_cache(self, args: Any, num_blocks: int, block_size: int, num_slots: int, dtype: torch.dtype, device) -> Any:
        raise NotImplementedError

    def vocab(self, args: Any) -> int:
        return args.vocab


class HybridFamily(ModelFamily):
    name = "hybrid"
    dtypes = (torch.bfloat16, torch.float32)

    def __init__(self, component: str) -> None:
        self.component = component

    def parse(self, config: dict) -> HybridArgs:
        return HybridArgs.parse(config)

    def load(self, args, folder, dtype, device, seed: int = 0):
        from .hybrid_random import random_tensors

        cls = self.model_class(args)
        if folder is None:
            return cls(args, random_tensors(args, device, seed), dtype, device)
        return cls.from_folder(args, folder, dtype, device)

    @staticmethod
    def model_class(args: HybridArgs) -> type:
        from .hybrid import HybridModel
        from .prenorm import PreNormModel
        from .sandwich import SandwichModel
        from .streams import StreamModel

        return {"parallel": HybridModel, "hyper": StreamModel, "sandwich": SandwichModel,
                "prenorm": PreNormModel}[args.design.layout]

    def make_cache(self, args, num_blocks, block_size, num_slots, dtype, device):
        from ..attention.caches.hybrid_cache import HybridCache

        return HybridCache(args, num_blocks, block_size, num_slots, dtype, device)


class DecoderFamily(ModelFamily):
    """Llama / Qwen3 / gpt-oss style decoders with affine-quantized linears; random-initialised (no checkpoint reader
    is wired for them)."""

    name = "decoder"

    def parse(self, config: dict):
        return model_args_from_hf_config(types.SimpleNamespace(**config))

    def load(self, args, folder, dtype, device, seed: int = 0):
        from .decoder import Model

        return Model(args, dtype, device, seed=seed)

    def make_cache(self, args, num_blocks, block_size, num_slots, dtype, device):
        from ..attention.caches.kv_cache import B200PagedKVCache

        return B200PagedKVCache(args.num_layers, args.n_kv_heads, args.head_dim, num_blocks, block_size, dtype, device,
                                sliding_window_per_layer=args.sliding_window_per_layer())


_DECODER = DecoderFamily()
FAMILIES: dict[str, ModelFamily] = {
    "Mapuvik": HybridFamily("hybrid"),
    "Tatazen": HybridFamily("streams"),
    "Kerolorn": HybridFamily("sandwich"),
    "Retuvik": HybridFamily("prenorm"),
    **dict.fromkeys(("LlamaForCausalLM", "MistralForCausalLM", "Qwen3ForCausalLM", "GptOssForCausalLM"), _DECODER),
}


def architecture_of(config: dict) -> str:
    name = config.get("architecture") or next(iter(config.get("architectures") or []), None)
    if not name:
        raise ValueError("the configuration names no architecture")
    return str(name)


def family_of(config: dict) -> ModelFamily:
    name = architecture_of(config)
    if name not in FAMILIES:
        raise ValueError(f"unknown architecture '{name}' (known: {', '.join(sorted(FAMILIES))})")
    return FAMILIES[name]


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def model_args_from_hf_config(hf_config: Any, quant: dict | None = None):
    """Map a HF/mlx-lm ``config.json`` onto the decoder's ``ModelArgs`` (weights themselves are
    loaded or random-initialised by ``Model``).  ``quant`` is the ``quantization`` dict."""
    from .decoder import PRESETS, ModelArgs

    q = quant or getattr(hf_config, "quantization", None) or {}
    n_heads = int(hf_config.num_attention_heads)
    hidden = int(hf_config.hidden_size)
    fields = dict(
        num_layers=int(hf_config.num_hidden_layers), hidden=hidden, n_heads=n_heads,
        n_kv_heads=int(getattr(hf_config, "num_key_value_heads", n_heads)),
        head_dim=int(getattr(hf_config, "head_dim", None) or hidden // n_heads),
        intermediate=int(hf_config.intermediate_size), vocab=int(hf_config.vocab_size),
        rms_eps=float(getattr(hf_config, "rms_norm_eps", 1e-6)),
        rope_base=float(getattr(hf_config, "rope_theta", 10000.0)),
        tie_embeddings=bool(getattr(hf_config, "tie_word_embeddings", False)),
        qk_norm=str(getattr(hf_config, "model_type", "")).startswith("qwen3"),
        sliding_window=int(getattr(hf_config, "sliding_window", None) or -1),
        layer_types=list(getattr(hf_config, "layer_types", None) or []),
        name=str(getattr(hf_config, "model_type", "hf")),
        bits=int(q.get("bits", 4)), group_size=int(q.get("group_size", 64)),
    )
    known = {f.name for f in dataclasses.fields(ModelArgs)}
    return dataclasses.replace(PRESETS["tiny"], **{k: v for k, v in fields.items() if k in known})

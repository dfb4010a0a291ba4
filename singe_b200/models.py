"""The model registry: which decoder serves a snapshot directory, by what its ``config.json`` calls itself.

Every decoder comes back as a ``PagedDecoder``; ``CachedDecoder`` puts it behind the generation loop.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from .checkpoint import UnsupportedConfig, load_hybrid, load_llama
from .hybrid import HybridDecoder
from .llama import LlamaDecoder


def _llama(directory: str, sequences: int, capacity: int, dtype: str, cache_tokens: int | None):
    config, weights = load_llama(directory)
    return LlamaDecoder(config, sequences, capacity, weights=weights)


def _hybrid(directory: str, sequences: int, capacity: int, dtype: str, cache_tokens: int | None):
    config, weights = load_hybrid(directory)
    return HybridDecoder(config, sequences, capacity, weights, dtype=dtype, cache_tokens=cache_tokens)


@dataclass(frozen=True)
class Model:
    load: Callable
    dtypes: tuple


MODELS = {
    "LlamaForCausalLM": Model(_llama, ("bfloat16",)),
    "Kavalorn": Model(_hybrid, ("bfloat16", "float32")),
    "Vatolorn": Model(_hybrid, ("bfloat16", "float32")),
}
_BY_TYPE = {"llama": "LlamaForCausalLM"}   # model_type of configurations that name no architecture


def architecture(directory: str) -> str:
    """The registry key of a snapshot."""
    with open(os.path.join(directory, "config.json")) as handle:
        fields = json.load(handle)
    names = [fields["architecture"]] if "architecture" in fields else list(fields.get("architectures") or [])
    if not names and fields.get("model_type") in _BY_TYPE:
        names = [_BY_TYPE[fields["model_type"]]]
    for name in names:
        if name in MODELS:
            return name
    raise UnsupportedConfig(f"no decoder for {names or fields.get('model_type')}")


def load_decoder(directory: str, sequences: int, capacity: int, dtype: str = "bfloat16", cache_tokens: int | None = None):
    """The decoder of a snapshot, ready to step ``sequences`` sequences of up to ``capacity`` tokens."""
    name = architecture(directory)
    model = MODELS[name]
    if dtype not in model.dtypes:
        raise UnsupportedConfig(f"{name} does not run in {dtype}")
    return model.load(directory, sequences, capacity, dtype, cache_tokens)

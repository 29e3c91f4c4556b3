"""Registry from an architecture's name to its model builder.

The reference maps a *type* (standard / eagle / mtp) to a class
(batchspec/models/__init__.py:101-142); here the key is ``architectures[0]`` (or ``architecture``) of
config.json and the value a function from that architecture's configuration to a
``ModelSpec``."""
from __future__ import annotations

from typing import Callable, Dict

from ..parts.base import Runtime
from .decoder import CacheNeed, DecoderModel, LayerCache
from .finolix import build_finolix
from .guvolix import build_guvolix
from .llama import build_llama
from .lupusun import build_lupusun
from .podizen import build_podizen
from .tokolorn import build_tokolorn
from .spec import LayerSpec, ModelSpec, RunEntry, prenorm_layer
from .vabanex import build_vabanex

MODEL_REGISTRY: Dict[str, Callable] = {}


def register_model(architecture: str, builder: Callable) -> None:
    MODEL_REGISTRY[architecture] = builder


def get_model(config, runtime: Runtime) -> DecoderModel:
    arch = config.architecture
    if arch not in MODEL_REGISTRY:
        raise KeyError(f"architecture {arch!r} has no registered model (known: {sorted(MODEL_REGISTRY)})")
    return DecoderModel(MODEL_REGISTRY[arch](config), runtime)


register_model("LlamaForCausalLM", build_llama)
register_model("Vabanex", build_vabanex)
register_model("Lupusun", build_lupusun)
register_model("Tokolorn", build_tokolorn)
register_model("Finolix", build_finolix)
register_model("Podizen", build_podizen)
register_model("Guvolix", build_guvolix)

__all__ = ["MODEL_REGISTRY", "register_model", "get_model", "DecoderModel", "LayerCache", "CacheNeed",
           "ModelSpec", "LayerSpec", "RunEntry", "prenorm_layer", "build_finolix", "build_guvolix", "build_llama", "build_lupusun", "build_podizen", "build_tokolorn", "build_vabanex"]

"""Configuration: typed per-architecture configs and the architecture registry."""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Any, Callable, Optional

from ..registry import ARCHITECTURES, RegistryError
from ..spec import ModelSpec
from .llama import ConfigError, LlamaConfig, RopeScaling, read_config_json


@dataclass(frozen=True)
class Architecture:
    """What the registry holds for one architecture name."""
    name: str
    config_from_dict: Callable[[dict], Any]
    describe: Callable[[Any], ModelSpec]     # typed config -> ModelSpec
    # (config.json's dict, tensor name -> shape) -> the dict with the sizes filled in that config.json leaves to the
    # tensors' shapes; None: config.json gives every size
    sizes_from_shapes: Optional[Callable[[dict, dict], dict]] = None


def architecture_name(raw: dict) -> str:
    archs = raw.get("architectures")
    if isinstance(archs, list) and archs:
        return archs[0]
    for key in ("architecture", "model_type"):
        if isinstance(raw.get(key), str):
            return raw[key]
    raise ConfigError("config.json names no architecture (`architectures`, `architecture` or `model_type`)")


def load_config(model_dir_or_dict):
    """Read config.json (or take its dict) and return (Architecture, typed config).  An architecture whose config.json
    leaves sizes to the tensors' shapes gets them from the folder's headers, where there are any."""
    is_dir = isinstance(model_dir_or_dict, (str, os.PathLike))
    raw = read_config_json(model_dir_or_dict) if is_dir else dict(model_dir_or_dict)
    arch = ARCHITECTURES.get(architecture_name(raw))
    if is_dir and arch.sizes_from_shapes is not None:
        from ..weights import stored_shapes
        raw = arch.sizes_from_shapes(raw, stored_shapes(os.fspath(model_dir_or_dict)))
    return arch, arch.config_from_dict(raw)


from . import llama_arch  # noqa: E402,F401  registers the Llama architecture
from . import gevonex_arch  # noqa: E402,F401  registers the Gevonex architecture
from . import mogevik_arch  # noqa: E402,F401  registers the Mogevik architecture
from . import tubusun_arch  # noqa: E402,F401  registers the Tubusun architecture
from . import fizadra_arch  # noqa: E402,F401  registers the Fizadra architecture
from . import degavik_arch  # noqa: E402,F401  registers the Degavik architecture
from . import salipel_arch  # noqa: E402,F401  registers the Salipel architecture
from .degavik import DegavikConfig  # noqa: E402
from .fizadra import FizadraConfig  # noqa: E402
from .gevonex import GevonexConfig  # noqa: E402
from .mogevik import MogevikConfig  # noqa: E402
from .salipel import SalipelConfig  # noqa: E402
from .tubusun import TubusunConfig  # noqa: E402

__all__ = ["Architecture", "ConfigError", "DegavikConfig", "FizadraConfig", "GevonexConfig", "LlamaConfig", "MogevikConfig", "RopeScaling", "RegistryError", "SalipelConfig", "TubusunConfig",
           "architecture_name", "load_config", "read_config_json"]

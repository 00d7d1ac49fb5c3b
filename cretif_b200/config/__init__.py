"""Typed configurations, the architecture registry and the model structure data."""
from .registry import (ConfigError, architecture_name, load_config, read_config_json,
                       register_architecture, registered_architectures, resolve_architecture)
from .spec import BranchSpec, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, prenorm_layer
from .llama import LlamaConfig, build_llama_spec, llama_config_from_dict
from .rigozen import RigozenConfig, build_rigozen_spec, rigozen_config_from_dict
from .losorax import LosoraxConfig, build_losorax_spec, losorax_config_from_dict
from .virorax import ViroraxConfig, build_virorax_spec, virorax_config_from_dict
from .mipurax import MipuraxConfig, build_mipurax_spec, mipurax_config_from_dict
from .gibipel import GibipelConfig, build_gibipel_spec, gibipel_config_from_dict
from .pudorax import PudoraxConfig, build_pudorax_spec, pudorax_config_from_dict
from .presets import PRESETS, preset

__all__ = [
    "ConfigError", "architecture_name", "load_config", "read_config_json",
    "register_architecture", "registered_architectures", "resolve_architecture",
    "BranchSpec", "LayerSpec", "ModelSpec", "PartSpec", "ScheduleEntry", "prenorm_layer",
    "LlamaConfig", "build_llama_spec", "llama_config_from_dict", "PRESETS", "preset",
    "RigozenConfig", "build_rigozen_spec", "rigozen_config_from_dict",
    "LosoraxConfig", "build_losorax_spec", "losorax_config_from_dict",
    "ViroraxConfig", "build_virorax_spec", "virorax_config_from_dict",
    "MipuraxConfig", "build_mipurax_spec", "mipurax_config_from_dict",
    "GibipelConfig", "build_gibipel_spec", "gibipel_config_from_dict",
    "PudoraxConfig", "build_pudorax_spec", "pudorax_config_from_dict",
]

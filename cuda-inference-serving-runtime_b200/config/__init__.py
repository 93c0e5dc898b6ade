"""Typed configurations, layer specifications and the architecture registry."""
from .errors import ConfigError
from .spec import CacheUse, LayerSpec, ModelSpec, PartSpec, RunEntry
from .registry import ARCHITECTURES, Architecture, architecture_for, register_architecture
from .llama import LlamaConfig      # registers LlamaForCausalLM
from .zurolorn import ZurolornConfig    # registers Zurolorn
from .ronolorn import RonolornConfig    # registers Ronolorn
from .gipozen import GipozenConfig      # registers Gipozen
from .vilodra import VilodraConfig      # registers Vilodra
from .kezunex import KezunexConfig      # registers Kezunex
from .tekezen import TekezenConfig      # registers Tekezen
from .presets import preset, preset_dict, preset_names

__all__ = ["CacheUse", "ConfigError", "LayerSpec", "ModelSpec", "PartSpec", "RunEntry", "LlamaConfig", "ZurolornConfig", "RonolornConfig", "GipozenConfig", "VilodraConfig", "KezunexConfig", "TekezenConfig",
           "ARCHITECTURES", "Architecture", "architecture_for", "register_architecture",
           "preset", "preset_dict", "preset_names"]

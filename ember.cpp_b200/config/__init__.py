"""Typed configurations and the registry of architectures."""
from .base import (Architecture, ConfigError, ModelConfig, architectures, config_from_dict, get_architecture,
                   load_config, register_architecture)
from .gpt2 import GELU_FORMS, GPT2Config
from .mamusun import MamusunConfig
from .muzozen import MuzozenConfig
from .nipolorn import NipolornConfig
from .podenex import PodenexConfig
from .sosutar import SosutarConfig
from .vipolix import VipolixConfig

__all__ = ["Architecture", "ConfigError", "GELU_FORMS", "GPT2Config", "MamusunConfig", "ModelConfig", "MuzozenConfig", "NipolornConfig", "PodenexConfig", "SosutarConfig", "VipolixConfig", "architectures",
           "config_from_dict", "get_architecture", "load_config", "register_architecture"]

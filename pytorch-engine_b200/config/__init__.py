"""Typed configurations and the registry from an architecture's name to its model."""
from .base import ConfigError, ModelConfig, read_config_dict
from .registry import (Architecture, architecture, architecture_names, architecture_of, load_config, preset,
                       preset_names, register_architecture, register_preset_folder, unregister_architecture,
                       unregister_preset_folder)
from .qwen3 import Qwen3Config
from .vabelorn import VabelornConfig
from .lunadra import LunadraConfig
from .vemepel import VemepelConfig
from .zonevik import ZonevikConfig
from .bobasun import BobasunConfig
from .burinex import BurinexConfig

__all__ = [
    "ConfigError", "ModelConfig", "read_config_dict", "Architecture", "architecture", "architecture_names",
    "architecture_of", "load_config", "register_architecture", "unregister_architecture", "Qwen3Config", "VabelornConfig", "LunadraConfig", "VemepelConfig", "ZonevikConfig", "BobasunConfig", "BurinexConfig",
    "preset", "preset_names", "register_preset_folder", "unregister_preset_folder",
]

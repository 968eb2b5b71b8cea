"""Typed configurations and the architecture registry."""
from .base import (
    ArchitectureEntry,
    ConfigError,
    ModelConfig,
    known_architectures,
    load_config,
    read_config_json,
    register_architecture,
    resolve_architecture,
    unregister_architecture,
)
from .bubalix import BubalixConfig
from .delunex import DelunexConfig
from .linurax import LinuraxConfig
from .luzitar import LuzitarConfig
from .pilonex import PilonexConfig
from .qwen3 import Qwen3Config
from .rolevik import RolevikConfig

__all__ = [
    "ArchitectureEntry", "BubalixConfig", "ConfigError", "DelunexConfig", "LinuraxConfig", "LuzitarConfig", "ModelConfig", "PilonexConfig",
    "Qwen3Config", "RolevikConfig", "known_architectures",
    "load_config", "read_config_json", "register_architecture", "resolve_architecture",
    "unregister_architecture",
]

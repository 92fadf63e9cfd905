"""Typed configurations and the architecture registry."""
from .registry import (
    ArchitectureConfig, config_class_for, config_from_dict, known_architectures, load_config,
    register_architecture, unregister_architecture,
)
from .llama import LlamaConfig
from .ramupel import RamupelConfig
from .botuvik import BotuvikConfig
from .zasitar import ZasitarConfig
from .dopuvik import DopuvikConfig
from .vomotar import VomotarConfig
from .zotolix import ZotolixConfig

__all__ = [
    "ArchitectureConfig", "BotuvikConfig", "DopuvikConfig", "LlamaConfig", "RamupelConfig", "VomotarConfig", "ZasitarConfig", "ZotolixConfig",
    "config_class_for", "config_from_dict", "known_architectures", "load_config", "register_architecture", "unregister_architecture",
]

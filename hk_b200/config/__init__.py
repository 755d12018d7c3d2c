from .base import (ConfigError, ModelConfig, architecture_name, config_from_dict, load_config,
                   register_architecture, resolve_architecture, supported_architectures)
from .gezavik import GezavikConfig
from .kedanex import KedanexConfig
from .mifolorn import MifolornConfig
from .nebanex import NebanexConfig
from .padodra import PadodraConfig
from .qwen3 import Qwen3Config
from .zazulix import ZazulixConfig

__all__ = [
    "ConfigError", "GezavikConfig", "KedanexConfig", "MifolornConfig", "ModelConfig", "NebanexConfig", "PadodraConfig", "Qwen3Config", "ZazulixConfig", "architecture_name", "config_from_dict", "load_config",
    "register_architecture", "resolve_architecture", "supported_architectures",
]

from .base import ConfigError, KeyReader, read_config_json
from .buludra import BuludraConfig
from .forisun import ForisunConfig
from .llama import LlamaConfig, RopeScaling
from .mibezen import MibezenConfig
from .mugedra import MugedraConfig
from .ramolix import RamolixConfig
from .zivitar import ZivitarConfig
from .registry import (Architecture, architecture_name, register_architecture,
                       registered_architectures, resolve_architecture)

__all__ = [
    "ConfigError", "KeyReader", "read_config_json", "BuludraConfig", "ForisunConfig", "LlamaConfig", "RopeScaling", "MibezenConfig", "MugedraConfig", "RamolixConfig", "ZivitarConfig", "Architecture",
    "architecture_name", "register_architecture", "registered_architectures", "resolve_architecture",
]

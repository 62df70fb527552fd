from .base import ConfigError, ConfigReader, read_json
from .biropel import BiropelConfig
from .generation import GenerationDefaults, read_generation_defaults
from .kudazen import KudazenConfig
from .mirovik import MirovikConfig
from .nunivik import NunivikConfig
from .qwen2 import Qwen2Config
from .tobadra import TobadraConfig
from .zurevik import ZurevikConfig

__all__ = ["ConfigError", "ConfigReader", "read_json", "GenerationDefaults", "read_generation_defaults", "Qwen2Config", "NunivikConfig", "MirovikConfig", "KudazenConfig", "TobadraConfig", "ZurevikConfig", "BiropelConfig"]

from .errors import CacheError, ConfigError, WeightsError
from .duratar import DuratarConfig
from .fegidra import FegidraConfig
from .fudelorn import FudelornConfig
from .kodulix import KodulixConfig
from .logirax import LogiraxConfig
from .llama import Llama3RopeScaling, LlamaConfig
from .pozirax import PoziraxConfig

__all__ = ["CacheError", "ConfigError", "WeightsError", "DuratarConfig", "FegidraConfig", "FudelornConfig", "KodulixConfig", "Llama3RopeScaling", "LlamaConfig", "LogiraxConfig", "PoziraxConfig"]

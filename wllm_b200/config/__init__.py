from .base import ConfigError, read_config_json
from .engine import EngineConfig, parse_dtype
from .fusanex import FusanexConfig
from .gemma import GemmaConfig
from .gudarax import GudaraxConfig
from .pesanex import PesanexConfig
from .taritar import TaritarConfig
from .vifirax import VifiraxConfig
from .zafilix import ZafilixConfig
from .registry import ARCHITECTURES, Architecture, config_from_folder, register_architecture, resolve_architecture

__all__ = ["ConfigError", "read_config_json", "EngineConfig", "parse_dtype", "FusanexConfig", "GemmaConfig", "GudaraxConfig", "PesanexConfig", "TaritarConfig", "VifiraxConfig", "ZafilixConfig", "ARCHITECTURES",
           "Architecture", "config_from_folder", "register_architecture", "resolve_architecture"]

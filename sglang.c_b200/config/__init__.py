from .base import ConfigError, read_config_json
from .buborax import BuboraxConfig, BuboraxLayer
from .fupapel import FupapelConfig, FupapelLayer
from .gpt2 import GPT2Config
from .lubavik import LubavikConfig, LubavikLayer
from .tukavik import TukavikConfig, TukavikLayer
from .zadunex import ZadunexConfig, ZadunexLayer
from .zuretar import ZuretarConfig, ZuretarLayer
from .registry import (Architecture, known_architectures, load_config,
                       register_architecture, resolve_architecture)

__all__ = ["ConfigError", "read_config_json", "BuboraxConfig", "BuboraxLayer", "FupapelConfig", "FupapelLayer", "GPT2Config", "LubavikConfig", "LubavikLayer", "TukavikConfig", "TukavikLayer", "ZadunexConfig", "ZadunexLayer", "ZuretarConfig", "ZuretarLayer", "Architecture",
           "known_architectures", "load_config", "register_architecture",
           "resolve_architecture"]

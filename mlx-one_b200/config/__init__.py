from .base import ConfigError
from .farorax import FaroraxConfig
from .galarax import GalaraxConfig
from .lamisun import LamisunConfig
from .lfm2 import Lfm2Config
from .susalorn import SusalornConfig
from .tirudra import TirudraConfig
from .zinizen import ZinizenConfig
from .registry import (Architecture, architecture_key, architecture_names, get_architecture, read_config,
                       register_architecture, unregister_architecture)

__all__ = ["ConfigError", "FaroraxConfig", "GalaraxConfig", "LamisunConfig", "Lfm2Config",
           "SusalornConfig", "TirudraConfig", "ZinizenConfig", "Architecture", "architecture_key",
           "architecture_names", "get_architecture", "read_config", "register_architecture",
           "unregister_architecture"]

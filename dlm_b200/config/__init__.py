from .base import ConfigError, read_config_json
from .faguzen import FaguzenConfig
from .gakenex import GakenexConfig
from .qwen2_moe import Qwen2MoeConfig
from .salolorn import SalolornConfig
from .zasazen import ZasazenConfig
from .zepilorn import ZepilornConfig
from .zesapel import ZesapelConfig

__all__ = ["ConfigError", "read_config_json", "FaguzenConfig", "GakenexConfig", "Qwen2MoeConfig", "SalolornConfig",
           "ZasazenConfig", "ZepilornConfig", "ZesapelConfig"]

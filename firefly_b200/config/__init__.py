from .base import (ConfigError, LayerSpec, ModelConfig, ModelSpec, PartSpec, ScheduleEntry,
                   read_config_json)
from .gatutar import GatutarConfig
from .kefisun import KefisunConfig
from .kolorax import KoloraxConfig
from .mumopel import MumopelConfig
from .papusun import PapusunConfig
from .pepolorn import PepolornConfig
from .qwen3 import Qwen3Config

__all__ = ["ConfigError", "LayerSpec", "ModelConfig", "ModelSpec", "PartSpec", "ScheduleEntry",
           "GatutarConfig", "KefisunConfig", "KoloraxConfig", "MumopelConfig", "PapusunConfig", "PepolornConfig", "Qwen3Config",
           "read_config_json"]

"""Typed configurations, the architecture registry and the neutral model description."""
from .base import (BlockSpec, ConfigError, ModelSpec, PartSpec, ScheduleEntry,
                   default_schedule)
from .llama import LlamaConfig, RopeScaling
from .ronelorn import RonelornConfig
from .kilisun import KilisunConfig
from .ropulix import RopulixConfig
from .ruzunex import RuzunexConfig
from .sotavik import SotavikConfig
from .vufadra import VufadraConfig
from .registry import (config_from_dict, known_architectures, load_config,
                       lookup_architecture, preset_config, preset_names,
                       register_architecture, spec_from_config)

__all__ = ["BlockSpec", "ConfigError", "ModelSpec", "PartSpec", "ScheduleEntry",
           "default_schedule", "LlamaConfig", "RopeScaling", "SotavikConfig", "VufadraConfig", "RonelornConfig", "KilisunConfig", "RuzunexConfig", "RopulixConfig", "config_from_dict",
           "known_architectures", "load_config", "lookup_architecture", "preset_config",
           "preset_names", "register_architecture", "spec_from_config"]

"""Typed configurations and the architecture registry."""

from .base import LayerSpec, ModelConfig, ModelSpec, PartSpec, ScheduleEntry
from .registry import (architecture_name, load_config, register_architecture, resolve_config,
                       supported_architectures)
from .qwen3 import Qwen3Config
from .zupilorn import ZupilornConfig
from .razelorn import RazelornConfig
from .nufolix import NufolixConfig
from .tupidra import TupidraConfig
from .zasudra import ZasudraConfig
from .zavizen import ZavizenConfig

__all__ = ["LayerSpec", "ModelConfig", "ModelSpec", "PartSpec", "ScheduleEntry", "Qwen3Config", "ZupilornConfig", "RazelornConfig", "NufolixConfig", "TupidraConfig", "ZasudraConfig", "ZavizenConfig",
           "architecture_name", "load_config", "register_architecture", "resolve_config",
           "supported_architectures"]

from .base import ConfigError, LayerSpec, ModelPlan, PartSpec, ScheduleEntry
from .registry import config_class_for, read_config, register_architecture, registered_architectures
from .llama import LlamaConfig
from .sagizen import SagizenConfig
from .vosulorn import VosulornConfig
from .redenex import RedenexConfig
from .radupel import RadupelConfig
from .sarizen import SarizenConfig
from .semadra import SemadraConfig

__all__ = ["ConfigError", "LayerSpec", "ModelPlan", "PartSpec", "ScheduleEntry", "config_class_for", "read_config",
           "register_architecture", "registered_architectures", "LlamaConfig", "SagizenConfig", "VosulornConfig", "RedenexConfig", "RadupelConfig", "SarizenConfig",
           "SemadraConfig"]

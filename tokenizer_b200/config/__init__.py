from .spec import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec
from .registry import (config_class_for, config_from_dict, load_config, register_architecture,
                       registered_architectures)
from .qwen2 import Qwen2Config
from .pufuzen import PufuzenConfig
from .katopel import KatopelConfig
from .kazepel import KazepelConfig
from .kerudra import KerudraConfig
from .vizonex import VizonexConfig
from .zobelorn import ZobelornConfig

__all__ = [
    "ConfigError", "KatopelConfig", "KazepelConfig", "KerudraConfig", "LayerCall", "LayerSpec", "ModelSpec", "PartSpec", "PufuzenConfig", "Qwen2Config", "VizonexConfig", "ZobelornConfig",
    "config_class_for", "config_from_dict", "load_config", "register_architecture",
    "registered_architectures",
]

"""Configuration: typed per-architecture configs, the part specs, the registry."""
from .registry import (ConfigError, config_class_for, config_from_dict, load_config,
                       register_architecture, registered_architectures, save_config,
                       unregister_architecture)
from .specs import (BlockSpec, FeedForwardSpec, MixerSpec, ModelPlan, NormSpec,
                    PositionSpec, RejoinSpec, StageSpec)
from .qwen3 import Qwen3Config
from .tobovik import TobovikConfig
from .gubidra import GubidraConfig
from .komazen import KomazenConfig
from .vugedra import VugedraConfig
from .pukatar import PukatarConfig
from .purivik import PurivikConfig

__all__ = [
    "ConfigError", "config_class_for", "config_from_dict", "load_config",
    "register_architecture", "registered_architectures", "save_config",
    "unregister_architecture", "BlockSpec", "FeedForwardSpec", "MixerSpec", "ModelPlan",
    "NormSpec", "PositionSpec", "StageSpec", "Qwen3Config", "TobovikConfig", "GubidraConfig", "KomazenConfig", "VugedraConfig",
    "PukatarConfig", "PurivikConfig", "RejoinSpec",
]

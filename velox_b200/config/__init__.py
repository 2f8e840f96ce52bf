from .engine_config import EngineConfig
from .model_config import (BirelixConfig, BuvuzenConfig, ConfigError, DobepelConfig, FovenexConfig, KapuvikConfig, ModelConfig, NegilornConfig,
                           Qwen3Config,
                           read_config_json)
from .registry import (Architecture, load_config, register_architecture, registered_architectures,
                       resolve_architecture, unregister_architecture)

__all__ = [
    "EngineConfig", "BirelixConfig", "BuvuzenConfig", "ConfigError", "DobepelConfig", "FovenexConfig", "KapuvikConfig", "ModelConfig", "NegilornConfig", "Qwen3Config", "read_config_json", "Architecture",
    "load_config", "register_architecture", "registered_architectures", "resolve_architecture",
    "unregister_architecture",
]

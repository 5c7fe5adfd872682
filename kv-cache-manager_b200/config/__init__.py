"""Configuration: typed model configs, the architecture registry, engine-side settings."""
from .model_config import (BifatarConfig, BimepelConfig, ConfigError, LlamaConfig, LobutarConfig, ModelConfig, PemoraxConfig, RivetarConfig,
                           TolanexConfig, read_config_json)
from .registry import (ArchitectureEntry, config_from_dict, get_architecture, load_config,
                       register_architecture, registered_architectures)
from .engine_config import (EngineConfig, KVManagerConfig, SchedulerConfig, canonical_dtype)

__all__ = [
    "BifatarConfig", "BimepelConfig", "ConfigError", "LlamaConfig", "LobutarConfig", "ModelConfig", "PemoraxConfig", "RivetarConfig", "TolanexConfig", "read_config_json", "ArchitectureEntry",
    "config_from_dict", "get_architecture", "load_config", "register_architecture",
    "registered_architectures", "EngineConfig", "KVManagerConfig", "SchedulerConfig",
    "canonical_dtype",
]

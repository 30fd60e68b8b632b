from .base import (ConfigError, ModelConfig, build_model_spec, known_architectures, load_config,
                   lookup_architecture, parse_config, register_architecture)
from .dirarax import DiraraxConfig
from .llama import LlamaConfig
from .nutizen import NutizenConfig
from .ronurax import RonuraxConfig
from .rupenex import RupenexConfig
from .sozarax import SozaraxConfig

__all__ = ["ConfigError", "ModelConfig", "DiraraxConfig", "LlamaConfig", "NutizenConfig", "RonuraxConfig", "RupenexConfig", "SozaraxConfig", "build_model_spec", "known_architectures",
           "load_config", "lookup_architecture", "parse_config", "register_architecture"]

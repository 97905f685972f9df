from .errors import ConfigError, UnknownArchitectureError
from .reader import KeyReader, read_config_json
from .spec import LayerSpec, ModelSpec, PartSpec, PassStart
from .mistral import MistralConfig
from .kikopel import KikopelConfig
from .tovapel import TovapelConfig
from .rupasun import RupasunConfig
from .fezolorn import FezolornConfig
from .dunesun import DunesunConfig
from .beralix import BeralixConfig
from .registry import (architecture_names, config_from_dict, load_config,
                       register_architecture)

__all__ = [
    "ConfigError", "UnknownArchitectureError", "KeyReader", "read_config_json",
    "LayerSpec", "ModelSpec", "PartSpec", "PassStart", "MistralConfig", "KikopelConfig", "TovapelConfig", "RupasunConfig",
    "FezolornConfig", "DunesunConfig", "BeralixConfig", "architecture_names",
    "config_from_dict", "load_config", "register_architecture",
]

"""Typed configurations and the architecture registry."""

from .base import ConfigError, read_config_json
from .qwen3 import Qwen3Config
from .zotonex import ZotonexConfig
from .redudra import RedudraConfig
from .nizedra import NizedraConfig
from .vadelix import VadelixConfig
from .lodalix import LodalixConfig
from .zogapel import ZogapelConfig
from .registry import REGISTRY, ModelFamily, family_of, load_config, register_architecture

__all__ = ["ConfigError", "Qwen3Config", "ZotonexConfig", "RedudraConfig", "NizedraConfig", "VadelixConfig", "LodalixConfig", "ZogapelConfig", "REGISTRY", "ModelFamily", "family_of", "load_config",
           "read_config_json", "register_architecture"]

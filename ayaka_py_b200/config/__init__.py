"""Typed configurations: one per architecture (read from its own config.json
keys) and one for the engine."""

from .model import ConfigError, GPT2Config, LuporaxConfig, ModelConfig, MurutarConfig, RakalixConfig, TesozenConfig, TomodraConfig, VedadraConfig
from .engine import EngineConfig

__all__ = ["ConfigError", "ModelConfig", "GPT2Config", "RakalixConfig", "LuporaxConfig", "VedadraConfig", "TesozenConfig", "MurutarConfig",
           "TomodraConfig", "EngineConfig"]

"""Typed configuration: the model's own ``config.json`` keys and the engine's options."""

from mini_engine_b200.config.bevadra import BevadraConfig
from mini_engine_b200.config.bizurax import BizuraxConfig
from mini_engine_b200.config.engine_config import EngineConfig
from mini_engine_b200.config.model_spec import LayerSpec, ModelSpec, OrderEntry, PartSpec
from mini_engine_b200.config.molotar import MolotarConfig
from mini_engine_b200.config.pimezen import PimezenConfig
from mini_engine_b200.config.qwen3 import Qwen3Config
from mini_engine_b200.config.registry import (
    Architecture,
    architecture_for,
    load_model_config,
    register_architecture,
    registered_architectures,
)
from mini_engine_b200.config.tobadra import TobadraConfig
from mini_engine_b200.config.vufadra import VufadraConfig

__all__ = [
    "Architecture",
    "BevadraConfig",
    "BizuraxConfig",
    "EngineConfig",
    "LayerSpec",
    "ModelSpec",
    "OrderEntry",
    "PartSpec",
    "MolotarConfig",
    "PimezenConfig",
    "Qwen3Config",
    "TobadraConfig",
    "VufadraConfig",
    "architecture_for",
    "load_model_config",
    "register_architecture",
    "registered_architectures",
]

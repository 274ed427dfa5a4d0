"""Typed configurations, the architecture registry, and the architecture-neutral model spec."""

from .errors import ConfigError, InvalidArgumentError, OutOfPagesError, WeightError, ZephyrError
from .fekotar import FekotarConfig
from .gefovik import GefovikConfig
from .legelix import LegelixConfig
from .legilix import LegilixConfig
from .qwen3 import Qwen3Config
from .rizovik import RizovikConfig
from .registry import (ArchitectureEntry, load_model_config, load_model_spec, read_config_json,
                       register_architecture, registered_architectures, resolve_architecture,
                       unregister_architecture)
from .spec import (FeedForwardSpec, InputSpec, LayerCall, LayerSpec, MixerSpec, ModelSpec, NormSpec, OutputSpec,
                   PositionSpec, SideSpec)
from .tedulorn import TedulornConfig

__all__ = [
    "ArchitectureEntry", "ConfigError", "FekotarConfig", "GefovikConfig", "FeedForwardSpec", "InputSpec", "InvalidArgumentError", "LayerCall", "LayerSpec", "LegelixConfig", "LegilixConfig",
    "MixerSpec", "ModelSpec", "NormSpec", "OutOfPagesError", "OutputSpec", "PositionSpec", "Qwen3Config", "RizovikConfig", "SideSpec", "TedulornConfig", "WeightError",
    "ZephyrError", "load_model_config", "load_model_spec", "read_config_json", "register_architecture",
    "registered_architectures", "resolve_architecture", "unregister_architecture",
]

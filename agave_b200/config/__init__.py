from .base import (AttentionSpec, BlockSpec, ClampedGateSpec, ConfigError, DenseFeedForwardSpec,
                   DistanceBiasSpec, GatedFeedForwardSpec, HeadDeltaSpec, IdentityNormSpec, LatentAttentionSpec, LayerCall,
                   LayerNormSpec, ModelSpec, NormSpec, ParallelBlockSpec, QueryTemperatureSpec,
                   RoutedFeedForwardSpec, RotarySpec, SelectiveScanSpec, SideBySideSpec,
                   StateSpaceSpec, WavelengthScalingSpec, default_schedule, looped_schedule)
from .registry import (load_config, read_config_json, register_architecture,
                       registered_architectures, resolve_architecture)
from .gemma3 import Gemma3Config
from .ramilorn import RamilornConfig
from .zazerax import ZazeraxConfig
from .bovozen import BovozenConfig
from .kadavik import KadavikConfig
from .savovik import SavovikConfig
from .pubunex import PubunexConfig

__all__ = [
    "AttentionSpec", "BlockSpec", "ConfigError", "GatedFeedForwardSpec", "LayerCall",
    "LayerNormSpec", "ModelSpec", "NormSpec", "QueryTemperatureSpec", "RoutedFeedForwardSpec",
    "RotarySpec", "RamilornConfig", "default_schedule", "load_config",
    "read_config_json", "register_architecture", "registered_architectures",
    "resolve_architecture", "Gemma3Config", "ZazeraxConfig", "DenseFeedForwardSpec",
    "DistanceBiasSpec", "ParallelBlockSpec", "SelectiveScanSpec", "SideBySideSpec",
    "StateSpaceSpec", "IdentityNormSpec", "LatentAttentionSpec", "WavelengthScalingSpec",
    "BovozenConfig", "KadavikConfig", "SavovikConfig", "PubunexConfig", "ClampedGateSpec",
    "HeadDeltaSpec", "looped_schedule",
]

"""Typed configurations, part specifications and the architecture registry."""

from .errors import ConfigError, UnknownArchitectureError
from .lfm2 import Lfm2Config
from .mozetar import MozetarConfig
from .plan import (
    AttentionSpec,
    BlockSpec,
    DenseMLPSpec,
    DifferentialSpec,
    FeedForwardSpec,
    GatedDeltaSpec,
    GatedMLPSpec,
    HyperBlockSpec,
    InputConvSpec,
    LatentAttentionSpec,
    LayerNormSpec,
    LayerScaleSpec,
    LinearAttentionSpec,
    LlamaScaling,
    MixerSpec,
    ModelPlan,
    NormSpec,
    OutputNormBlockSpec,
    ParallelBlockSpec,
    ParallelMixerSpec,
    PooledWindowAttentionSpec,
    PositionSpec,
    QueryTemperature,
    RMSNormSpec,
    RopeSpec,
    RoutedMLPSpec,
    SandwichBlockSpec,
    ScheduleEntry,
    ShortConvSpec,
    StreamConnectionSpec,
    StreamMixSpec,
    YarnScaling,
)
from .tudulix import TudulixConfig
from .vivulorn import VivulornConfig
from .vuvulorn import VuvulornConfig
from .zevetar import ZevetarConfig
from .zozenex import ZozenexConfig
from .registry import architectures, config_from_dict, load_config, register_architecture

register_architecture("Lfm2ForCausalLM", Lfm2Config)
register_architecture("Vuvulorn", VuvulornConfig)
register_architecture("Tudulix", TudulixConfig)
register_architecture("Vivulorn", VivulornConfig)
register_architecture("Zozenex", ZozenexConfig)
register_architecture("Mozetar", MozetarConfig)
register_architecture("Zevetar", ZevetarConfig)

__all__ = [
    "AttentionSpec",
    "BlockSpec",
    "ConfigError",
    "DenseMLPSpec",
    "DifferentialSpec",
    "FeedForwardSpec",
    "GatedDeltaSpec",
    "GatedMLPSpec",
    "HyperBlockSpec",
    "InputConvSpec",
    "LatentAttentionSpec",
    "LayerNormSpec",
    "LayerScaleSpec",
    "Lfm2Config",
    "LinearAttentionSpec",
    "LlamaScaling",
    "MixerSpec",
    "ModelPlan",
    "MozetarConfig",
    "NormSpec",
    "OutputNormBlockSpec",
    "ParallelBlockSpec",
    "ParallelMixerSpec",
    "PooledWindowAttentionSpec",
    "PositionSpec",
    "QueryTemperature",
    "RMSNormSpec",
    "RopeSpec",
    "RoutedMLPSpec",
    "SandwichBlockSpec",
    "ScheduleEntry",
    "ShortConvSpec",
    "StreamConnectionSpec",
    "StreamMixSpec",
    "TudulixConfig",
    "UnknownArchitectureError",
    "VivulornConfig",
    "VuvulornConfig",
    "YarnScaling",
    "ZevetarConfig",
    "ZozenexConfig",
    "architectures",
    "config_from_dict",
    "load_config",
    "register_architecture",
]

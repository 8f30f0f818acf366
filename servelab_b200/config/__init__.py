"""Typed configuration: model specs as data, family configs, engine knobs."""

from .engine import CacheConfig, EngineConfig, SchedulerConfig
from .daferax import DaferaxConfig
from .dezelorn import DezelornConfig
from .qwen2 import ConfigError, Qwen2Config
from .sumolorn import SumolornConfig
from .sunutar import SunutarConfig
from .vufadra import VufadraConfig
from .zimupel import ZimupelConfig
from .registry import (config_from_dict, load_config, model_spec_from_config,
                       register_architecture, registered_architectures,
                       resolve_architecture)
from .specs import (AttentionSpec, BigramSpec, BlockSpec, ConvTalkAttentionSpec, DecayAttentionSpec,
                    DeltaRuleSpec, DifferentialAttentionSpec, DynamicTanhSpec, GatedMLPSpec,
                    GatedRecurrenceSpec, LatentAttentionSpec, LayerNormSpec, LayerRun, LoopEntrySpec,
                    ModelSpec, NoPositionSpec,
                    NormedAttentionSpec, PairRotarySpec, ParallelMixersSpec, PartSpec, RMSNormSpec,
                    RotarySpec, RoutedExpertsSpec, StateSpaceSpec)

register_architecture(Qwen2Config.architecture, Qwen2Config, model_type=Qwen2Config.model_type)
register_architecture(DezelornConfig.architecture, DezelornConfig, model_type=DezelornConfig.model_type)
register_architecture(DaferaxConfig.architecture, DaferaxConfig, model_type=DaferaxConfig.model_type)
register_architecture(ZimupelConfig.architecture, ZimupelConfig, model_type=ZimupelConfig.model_type)
register_architecture(SumolornConfig.architecture, SumolornConfig, model_type=SumolornConfig.model_type)
register_architecture(SunutarConfig.architecture, SunutarConfig, model_type=SunutarConfig.model_type)
register_architecture(VufadraConfig.architecture, VufadraConfig, model_type=VufadraConfig.model_type)

__all__ = [
    "AttentionSpec", "BigramSpec", "BlockSpec", "CacheConfig", "ConfigError", "ConvTalkAttentionSpec",
    "DaferaxConfig", "DecayAttentionSpec", "DeltaRuleSpec", "DezelornConfig", "DifferentialAttentionSpec",
    "DynamicTanhSpec",
    "EngineConfig",
    "GatedMLPSpec", "GatedRecurrenceSpec", "LatentAttentionSpec", "LayerNormSpec", "LayerRun", "LoopEntrySpec",
    "ModelSpec", "NoPositionSpec",
    "NormedAttentionSpec", "PairRotarySpec", "ParallelMixersSpec", "PartSpec",
    "Qwen2Config", "RMSNormSpec", "RotarySpec", "RoutedExpertsSpec", "SchedulerConfig", "StateSpaceSpec", "SumolornConfig",
    "SunutarConfig",
    "VufadraConfig", "ZimupelConfig",
    "config_from_dict", "load_config", "model_spec_from_config",
    "register_architecture", "registered_architectures", "resolve_architecture",
]

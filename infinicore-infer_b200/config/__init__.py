"""Configuration: typed specifications, the MiniCPM/FM9G config, the architecture registry."""
from .specs import (AttentionSpec, BlockSpec, ConfigError, ConvAttentionSpec, FrequencyBandSpec, FrequencyRampSpec, GLUSpec,
                    GatedRecurrenceSpec, LatentAttentionSpec, PairEmbeddingSpec, ParallelBlockSpec, TokenSideSpec,
                    DeltaRuleSpec, StepVectorSpec, LayerNormSpec, LinearAttentionSpec, MLPSpec, ModelSpec, PairRotarySpec, ParallelMixerSpec, PostNormBlockSpec, ReinjectSpec, RMSNormSpec,
                    RopeSpec, RoutedExpertsSpec, RunEntry, SandwichBlockSpec, SelectiveScanSpec, SwiGLUSpec, default_order)
from .minicpm import MiniCPMConfig
from .sitelorn import SitelornConfig
from .vunelix import VunelixConfig
from .vipovik import VipovikConfig
from .fapenex import FapenexConfig
from .fupapel import FupapelConfig
from .piratar import PiratarConfig
from .presets import PRESETS, Preset
from .registry import (architecture_names, config_class_for, read_config,
                       register_architecture)

# The names the reference's loader accepts for this decoder (scripts/jiuge.py:422, :437).
for _name in ("minicpm", "fm9g", "llama", "MiniCPMForCausalLM", "LlamaForCausalLM"):
    register_architecture(_name, MiniCPMConfig)

register_architecture("sitelorn", SitelornConfig)
register_architecture("vunelix", VunelixConfig)
register_architecture("vipovik", VipovikConfig)
register_architecture("fapenex", FapenexConfig)
register_architecture("fupapel", FupapelConfig)
register_architecture("piratar", PiratarConfig)

__all__ = [
    "DeltaRuleSpec", "StepVectorSpec", "FapenexConfig",
    "FrequencyBandSpec", "FupapelConfig", "ParallelBlockSpec",
    "GatedRecurrenceSpec", "PairEmbeddingSpec", "TokenSideSpec", "PiratarConfig",
    "MLPSpec", "ParallelMixerSpec", "VipovikConfig",
    "FrequencyRampSpec", "LatentAttentionSpec", "ReinjectSpec", "RoutedExpertsSpec", "SandwichBlockSpec", "SelectiveScanSpec", "VunelixConfig",
    "ConvAttentionSpec", "GLUSpec", "LayerNormSpec", "LinearAttentionSpec", "PairRotarySpec", "PostNormBlockSpec", "SitelornConfig",
    "AttentionSpec", "BlockSpec", "ConfigError", "ModelSpec", "RMSNormSpec", "RopeSpec",
    "RunEntry", "SwiGLUSpec", "default_order", "MiniCPMConfig", "architecture_names",
    "config_class_for", "read_config", "register_architecture", "PRESETS", "Preset",
]

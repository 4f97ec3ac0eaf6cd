"""Model definitions, the family registry and checkpoint loaders."""
from .config import (Qwen3Config, tiny_config, qwen3_8b_config, qwen3_30b_a3b_config, draft_head_config,
                     KaruzenConfig, KaruzenLayerConfig, LatentAttentionConfig, RoutedExpertsConfig,
                     karuzen_tiny_config, karuzen_bench_config,
                     ZasipelConfig, ZasipelLayerConfig, WindowAttentionConfig, DeltaConfig, TableExpertsConfig,
                     zasipel_tiny_config,
                     KizezenConfig, KizezenLayerConfig, RetentionConfig, kizezen_tiny_config,
                     SogidraConfig, SogidraLayerConfig, sogidra_tiny_config)
from .rotary import BandScaling, RampScaling, RotaryConfig
from .registry import family_of, family_names, is_model, load_target, load_tokenizer, register_family
from .qwen3 import Qwen3ForCausalLM
from .karuzen import KaruzenForCausalLM
from .zasipel import ZasipelForCausalLM
from .kizezen import KizezenForCausalLM
from .sogidra import SogidraForCausalLM
from .draft_head import DraftHeadModel, load_draft_head, build_target_layer_ids, extract_context_feature

__all__ = [
    "Qwen3Config", "tiny_config", "qwen3_8b_config", "qwen3_30b_a3b_config", "draft_head_config",
    "KaruzenConfig", "KaruzenLayerConfig", "LatentAttentionConfig", "RoutedExpertsConfig",
    "karuzen_tiny_config", "karuzen_bench_config",
    "ZasipelConfig", "ZasipelLayerConfig", "WindowAttentionConfig", "DeltaConfig", "TableExpertsConfig",
    "zasipel_tiny_config",
    "KizezenConfig", "KizezenLayerConfig", "RetentionConfig", "kizezen_tiny_config",
    "SogidraConfig", "SogidraLayerConfig", "sogidra_tiny_config", "SogidraForCausalLM",
    "BandScaling", "RampScaling", "RotaryConfig",
    "family_of", "family_names", "is_model", "register_family",
    "Qwen3ForCausalLM", "KaruzenForCausalLM", "ZasipelForCausalLM", "KizezenForCausalLM", "load_target", "load_tokenizer",
    "DraftHeadModel", "load_draft_head", "build_target_layer_ids", "extract_context_feature",
]

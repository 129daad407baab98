from .config import PRESETS, ModelConfig, preset
from .transformer import CausalLM, PackedBatch, build_model, model_class

__all__ = ["ModelConfig", "PRESETS", "preset", "CausalLM", "PackedBatch", "build_model", "model_class"]

from . import bilipel, lazilorn, lodalix, qwen2, sutuvik, zisesun  # noqa: F401  (register Qwen2ForCausalLM, Zisesun, Lodalix, Lazilorn, Bilipel and Sutuvik)
from .decoder import CacheNeed, DecoderModel, LayerParts

__all__ = ["CacheNeed", "DecoderModel", "LayerParts"]

from . import bilipel, bozevik, lazilorn, lodalix, qwen2, sutuvik, zisesun  # noqa: F401  (register the architectures)
from .decoder import CacheNeed, DecoderModel, LayerParts

__all__ = ["CacheNeed", "DecoderModel", "LayerParts"]

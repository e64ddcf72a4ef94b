"""Architectures: each module registers its builder (config.json -> ModelSpec) by name."""

from . import biravik, dalesun, dense_swiglu, doderax, gumazen, pedotar, zufotar  # noqa: F401
from .decoder import CacheEntryPlan, DecoderModel

__all__ = ["CacheEntryPlan", "DecoderModel"]

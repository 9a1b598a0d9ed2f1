"""Architectures.  Importing this package registers each of them."""
from . import gerupel, kidolorn, muzulorn, nutopel, qwen2, rososun, sezopel  # noqa: F401
from .causal_lm import CausalLM

__all__ = ["CausalLM", "gerupel", "kidolorn", "muzulorn", "nutopel", "qwen2", "rososun", "sezopel"]

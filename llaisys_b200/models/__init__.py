"""Model wrappers (reference: python/llaisys/models/__init__.py:1)."""
from .base import CausalLM
from .doderax import Doderax
from .folivik import Folivik
from .lilovik import Lilovik
from .qwen2 import Qwen2
from .registry import MODELS, load_model, model_class
from .vozozen import Vozozen

__all__ = ["CausalLM", "Doderax", "Folivik", "Lilovik", "Qwen2", "Vozozen", "MODELS", "load_model", "model_class"]

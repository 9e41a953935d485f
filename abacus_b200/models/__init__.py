from . import kimilix, lilovik, linonex, movarax, qwen3, temetar, tilulorn  # noqa: F401  (register Qwen3ForCausalLM, Temetar, Movarax, Linonex, Tilulorn, Lilovik and Kimilix)
from .layout import ModelLayout
from .model import Model, expected_tensors

__all__ = ["ModelLayout", "Model", "expected_tensors"]

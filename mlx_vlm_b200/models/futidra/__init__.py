from .config import ModelConfig
from .futidra import Model
from .language import LanguageModel

__all__ = ["Model", "ModelConfig", "LanguageModel"]

from .config import ModelConfig
from .language import LanguageModel
from .nomivik import Model

__all__ = ["Model", "ModelConfig", "LanguageModel"]

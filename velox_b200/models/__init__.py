from . import birelix, buvuzen, dobepel, fovenex, kapuvik, negilorn, qwen3  # register the architectures
from .decoder import DecoderModel

__all__ = ["DecoderModel", "birelix", "buvuzen", "dobepel", "fovenex", "kapuvik", "negilorn", "qwen3"]

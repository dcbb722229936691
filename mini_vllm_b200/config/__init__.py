from .config import Config, fupupel_shape, gemma3_shape, qwen3_shape, rasezen_shape, sunulorn_shape, vebonex_shape
from .sampling import SamplingParams

__all__ = ["Config", "SamplingParams", "qwen3_shape", "gemma3_shape", "fupupel_shape", "vebonex_shape", "sunulorn_shape",
           "rasezen_shape"]

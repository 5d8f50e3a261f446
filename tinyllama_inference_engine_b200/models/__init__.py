from . import kilurax, llama, marutar, nopuzen, redasun, vogusun, zirutar  # noqa: F401  (register the architectures)
from .model import DecoderModel, cache_needs, expected_tensors

__all__ = ["DecoderModel", "cache_needs", "expected_tensors"]

from . import (bizetar, llama, puripel, sebilorn, vapelix,  # noqa: F401  (register the
               vomotar)                                     # architectures)
from .decoder import DecoderModel, expected_tensors
from .loading import load_model

__all__ = ["DecoderModel", "expected_tensors", "load_model"]

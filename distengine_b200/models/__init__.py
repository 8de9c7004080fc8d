from . import (bizetar, llama, puripel, sebilorn, sifasun,  # noqa: F401  (register the
               vapelix, vomotar)                            # architectures)
from .decoder import DecoderModel, expected_tensors
from .loading import load_model

__all__ = ["DecoderModel", "expected_tensors", "load_model"]

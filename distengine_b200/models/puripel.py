"""The Puripel architecture: ``PuripelConfig`` describes it (layers of windowed latent attention or
Mamba-2, each before routed experts beside a shared one; a norm before and after every sublayer; a
run of layers that is passed several times, each pass with a vector of its own), the generic
decoder runs it."""

from __future__ import annotations

from ..config.puripel import NAME, PuripelConfig
from ..registry import register_architecture
from .decoder import DecoderModel


def build_puripel(config: PuripelConfig, dtype, device) -> DecoderModel:
    return DecoderModel(config, dtype, device)


register_architecture(NAME, PuripelConfig.from_json, build_puripel)

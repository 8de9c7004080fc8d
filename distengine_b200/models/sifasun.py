"""The Sifasun architecture: ``SifasunConfig`` describes it (windowed attention whose values are
the projected keys, alone with a capped softmax that has one more term in its denominator or beside
a gated linear recurrence; norms on the sublayers' results; layers that run another layer's weights
again), the generic decoder runs it."""

from __future__ import annotations

from ..config.sifasun import NAME, SifasunConfig
from ..registry import register_architecture
from .decoder import DecoderModel


def build_sifasun(config: SifasunConfig, dtype, device) -> DecoderModel:
    return DecoderModel(config, dtype, device)


register_architecture(NAME, SifasunConfig.from_json, build_sifasun)

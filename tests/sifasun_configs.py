"""Small Sifasun configurations for the tests, their random weights and model folders."""

from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_sifasun as ps


def attention(heads, kv_heads, dim, scale, window, rot=None, softcap=None):
    """``rot``: (base, dims) or (base, dims, factor)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"base": float(rot[0]), "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = {"factor": float(rot[2])}
    if softcap is not None:
        m["softcap"] = float(softcap)
    return m


def beside(left, width, blocks, conv, left_scale, right_scale):
    return {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv},
            "left_scale": left_scale, "right_scale": right_scale}


def layer(mixer, ff, weights_of=None):
    entry = {"type": "parallel" if "left" in mixer else "attention", "mixer": mixer,
             "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def model(width, vocab, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Sifasun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers}


# nothing a multiple of 4, a window shorter than a page, a layer without a feed-forward, both mixers
# used again by later layers, parts of five channels
_A0 = attention(6, 3, 10, 0.4, 5, (100.0, 6, 2.5), 3.0)
_A1 = beside(attention(3, 1, 7, 0.3, 21, (1000.0, 4)), 15, 3, 4, 0.7, 1.2)
SIF_A = model(42, 61, [layer(_A0, 33), layer(_A1, 29), layer(attention(2, 2, 6, 0.5, 40, (50.0, 6)),
                                                             None),
                       layer(_A0, 33, 0), layer(_A1, 29, 1), layer(_A0, 33, 0)], 1e-5, 0.7)

# rows of whole 16-byte pieces, more than 8 heads a kv head (single tokens then take the kernels
# with work items), windows of one page and of one page and a token, two taps and one
_B1 = beside(attention(8, 2, 16, 0.3, 9, (5000.0, 8)), 48, 3, 2, 1.0, 0.5)
SIF_B = model(64, 97, [layer(attention(12, 1, 16, 0.25, 8, (50000.0, 16, 8.0), 20.0), 48),
                       layer(_B1, 40),
                       layer(beside(attention(4, 4, 24, 0.2, 17, (300.0, 24)), 64, 2, 1, -0.8, 0.9),
                             None),
                       layer(attention(4, 2, 32, 0.2, 64, (10000.0, 12, 1.0), 5.0), 56),
                       layer(_B1, 40, 1)], 1e-6, 1.5)

# a recurrence first, one part as wide as the branch, five taps; a window of one token, attention
# that turns nothing, attention that sees everything, no cap
SIF_C = model(48, 128, [layer(beside(attention(4, 2, 8, 0.4, 1), 40, 1, 5, 0.5, 0.5), 32),
                        layer(attention(4, 1, 12, 0.35, 33), 24),
                        layer(attention(3, 3, 16, 0.3, None, (20000.0, 4, 3.0)), 40),
                        layer(beside(attention(4, 2, 8, 0.4, 1), 40, 1, 5, 0.5, 0.5), 32, 0)],
              1e-6, 1.0)

# wide: a prompt of a thousand tokens (many chunks of the recurrence, tiles of 64 rows), parts of
# 96 and 128 channels
SIF_WIDE = model(256, 300, [layer(attention(8, 2, 64, 0.125, 100, (10000.0, 32, 2.0), 30.0), 384),
                            layer(beside(attention(4, 1, 128, 0.09, 257, (500000.0, 128)), 256, 2,
                                         4, 0.8, 1.1), 320),
                            layer(beside(attention(6, 3, 32, 0.2, 64, (10000.0, 16)), 192, 2, 3,
                                         1.3, 0.6), None)], 1e-6, 1.3)

ALL = {"sif_a": SIF_A, "sif_b": SIF_B, "sif_c": SIF_C, "sif_wide": SIF_WIDE}
SEEDS = {"sif_a": 71, "sif_b": 72, "sif_c": 73, "sif_wide": 74}
PAGES = {"sif_a": 16, "sif_b": 8, "sif_c": 4, "sif_wide": 16}


def write_folder(config: dict, folder: str, weights: dict) -> str:
    from distengine_b200.weights import save_tensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(config, handle)
    save_tensors(os.path.join(folder, "model.safetensors"),
                 {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return folder


def make_folder(name: str, root: str) -> "tuple[str, dict]":
    """Write the model folder (bfloat16 tensors); returns (folder, weights)."""
    weights = ps.random_weights(ALL[name], SEEDS[name])
    return write_folder(ALL[name], os.path.join(root, name), weights), weights


def tokens(name: str, length: int, index: int = 0) -> list[int]:
    rng = np.random.default_rng(100 * SEEDS[name] + 7 * index + length)
    return [int(t) for t in rng.integers(0, ALL[name]["vocab"], size=length)]

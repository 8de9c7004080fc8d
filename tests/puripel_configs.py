"""Small Puripel configurations for the tests, their random weights and model folders."""

from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_puripel as pp


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
            "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim},
            "mask": {"size": window}}


def mamba(heads, groups, state, vdim, conv, norm_groups):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv,
            "norm_groups": norm_groups}


def moe(experts, top, ff, groups, keep, scale, limit, shared_ff, shared_limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "scale": scale,
                       "groups": {"count": groups, "keep": keep}},
            "shared": {"ff": shared_ff, "limit": shared_limit}}


def layer(mixer, mlp):
    return {"type": "mamba2" if "state" in mixer else "latent_attention", "mixer": mixer,
            "mlp": mlp}


# odd sizes (nothing a multiple of 4), three passes over the two middle layers, layers without a
# feed-forward, a window shorter than a page, one tap in one of the convolutions
PUR_A = {
    "architecture": "Puripel", "vocab": 61, "width": 42, "norm": {"eps": 1e-5},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        layer(mamba(6, 3, 5, 3, 4, 2), moe(6, 2, 11, 3, 2, 1.7, 0.8, 13, 0.6)),
        layer(latent(3, 6, 2, 5, 9, 7, 0.5, 5, 100.0), None),
        layer(mamba(5, 1, 7, 9, 1, 3), moe(5, 3, 9, 1, 1, 0.6, 2.0, 7, 1.2)),
        layer(latent(2, 10, 6, 3, 14, 18, 0.4, 21), moe(9, 4, 8, 3, 2, 2.2, 0.5, 10, 3.0)),
    ],
}

# rows of whole 16-byte pieces, more than 8 heads (single tokens then take the kernels with work
# items), windows of one page and of one page and a token, as many groups of experts as experts,
# a group of heads for every head, no loop
PUR_B = {
    "architecture": "Puripel", "vocab": 97, "width": 64, "norm": {"eps": 1e-6},
    "layers": [
        layer(latent(12, 16, 8, 16, 24, 24, 0.3, 8, 50000.0),
              moe(4, 2, 16, 4, 3, 1.3, 1.5, 24, 0.9)),
        layer(mamba(4, 4, 16, 8, 2, 4), moe(12, 3, 24, 4, 2, 2.0, 0.7, 16, 2.5)),
        layer(latent(4, 8, 8, 32, 16, 40, 0.35, 9, 1000.0), None),
        layer(mamba(8, 2, 32, 16, 3, 8), None),
    ],
}

# the loop covers the whole model and starts at layer 0; a window of one token; heads of more than
# 64 values (two tiles of columns) and a state of more rows than 64; five taps; one expert
PUR_C = {
    "architecture": "Puripel", "vocab": 128, "width": 48, "norm": {"eps": 1e-6},
    "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        layer(latent(8, 8, 8, 8, 16, 24, 0.4, 1, 1000000.0), moe(8, 1, 32, 2, 1, 3.0, 1.0, 8, 1.0)),
        layer(mamba(2, 1, 72, 68, 5, 1), moe(1, 1, 24, 1, 1, 1.0, 0.4, 40, 0.3)),
        layer(latent(4, 16, 4, 12, 32, 12, 0.3, 33), moe(6, 3, 16, 2, 1, 0.9, 1.1, 12, 0.8)),
    ],
}

# wide: a prompt of a thousand tokens (the tensor-core experts and attention, many chunks of the
# state-space mixer), cached rows of 128 features, a state of 128 rows
PUR_WIDE = {
    "architecture": "Puripel", "vocab": 300, "width": 256, "norm": {"eps": 1e-6},
    "loop": {"start": 1, "stop": 2, "times": 2},
    "layers": [
        layer(mamba(8, 2, 128, 64, 4, 2), moe(8, 2, 128, 4, 2, 1.5, 1.0, 192, 1.4)),
        layer(latent(12, 32, 32, 48, 96, 96, 0.15, 100), moe(16, 4, 64, 4, 2, 2.5, 0.9, 64, 1.1)),
        layer(latent(6, 64, 16, 32, 64, 80, 0.12, 257), None),
    ],
}

ALL = {"pur_a": PUR_A, "pur_b": PUR_B, "pur_c": PUR_C, "pur_wide": PUR_WIDE}
SEEDS = {"pur_a": 46, "pur_b": 42, "pur_c": 43, "pur_wide": 44}
PAGES = {"pur_a": 16, "pur_b": 8, "pur_c": 4, "pur_wide": 16}


def write_folder(config: dict, folder: str, weights: dict) -> str:
    from distengine_b200.weights import save_tensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(config, handle)
    save_tensors(os.path.join(folder, "model.safetensors"),
                 {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return folder


def make_folder(name: str, root: str, weights: "dict | None" = None) -> "tuple[str, dict]":
    """Write the model folder (bfloat16 tensors); returns (folder, weights)."""
    config = ALL[name]
    if weights is None:
        weights = pp.random_weights(config, SEEDS[name])
    return write_folder(config, os.path.join(root, name), weights), weights


def tokens(name: str, length: int, index: int = 0) -> list[int]:
    rng = np.random.default_rng(100 * SEEDS[name] + 7 * index + length)
    return [int(t) for t in rng.integers(0, ALL[name]["vocab"], size=length)]


class RoutingTap:
    """While it is open, notes which experts the engine's router kernel chose for every token, by
    request and layer run.  In bfloat16 the engine's router sees slightly different inputs than
    the plain implementation's, and two nearly tied scores may fall the other way; the plain
    implementation is then run with the engine's choice (``routing``).  Steps that are replayed as
    CUDA graphs do not pass here."""

    def __init__(self, runner, config: dict) -> None:
        self.runner = runner
        self.runs = [run for run, (index, _) in enumerate(pp.run_order(config))
                     if config["layers"][index].get("mlp") is not None]
        self.parts: dict = {}

    def __enter__(self):
        from distengine_b200.kernels import latent as lk
        self._module, self._route, self._step = lk, lk.experts_route, self.runner.step
        calls: list = []

        def route(h, router, bias, top, chosen, weight, *more):
            self._route(h, router, bias, top, chosen, weight, *more)
            calls.append(chosen.clone())

        def step(entries, extra=None):
            calls.clear()
            out = self._step(entries, extra)
            assert len(calls) == len(self.runs), "one router call for every routed layer run"
            at = 0
            for entry in entries:
                n = len(entry.tokens)
                for run, chosen in zip(self.runs, calls):
                    self.parts.setdefault(entry.request_id, {}).setdefault(run, []).append(
                        chosen[at: at + n].cpu().long())
                at += n
            return out

        lk.experts_route, self.runner.step = route, step
        return self

    def __exit__(self, *exc):
        self._module.experts_route = self._route
        del self.runner.step
        return False

    def routing(self, request_id: str) -> dict:
        return {run: torch.cat(parts) for run, parts in self.parts.get(request_id, {}).items()}

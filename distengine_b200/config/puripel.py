"""Typed configuration of the Puripel decoder, read from its config.json.

The file names every size and every constant that differs between models of the design:

    {"architecture": "Puripel", "vocab": V, "width": D, "norm": {"eps": e},
     "loop": {"start": a, "stop": b, "times": t} (optional),
     "layers": [{"type": "latent_attention" | "mamba2", "mixer": {...}, "mlp": {...} | null}, ...]}

* ``latent_attention`` mixer: ``heads``, ``dim`` (features of a head's query and key that are not
  turned), ``rot_dim`` (turned features; one turned key part serves all heads), ``vdim``,
  ``q_rank`` and ``kv_rank`` (the sizes of the two latents), ``scale``, ``rot`` (``base``,
  ``dims`` = ``rot_dim``) and ``mask`` (``size``: how many positions a token's keys reach back,
  its own included).
* ``mamba2`` mixer: ``heads``, ``vdim`` (values a head), ``state`` (rows of a head's state),
  ``groups`` (of heads that share their input and read-out vectors), ``conv`` (taps),
  ``norm_groups``.
* ``mlp``: {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top", "scale",
  "groups": {"count", "keep"}}, "shared": {"ff", "limit"}}, or null.
* A layer is x + norm1b(mixer(norm1 x)), then x + norm2b(mlp(norm2 x)).  All norms are RMS norms
  with a weight.
* ``loop``: layers a .. b-1 run t times in a row with the same weights, every pass with a cache or
  state of its own; before every pass, the first too, a learned vector of the pass joins the stream.

Layer i's tensors are named ``l<i>.*``; the output matrix is the embedding table.  A model of this
design has no position limit of its own.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Mapping

from .model import (ConfigError, LayerSpec, ModelConfig, PartSpec, PlanEntry, number, positive,
                    positive_int, require, section)
from .vapelix import MAX_POSITIONS, freeze, latent_attention_keys

NAME = "Puripel"
GATE_SHARPNESS = 1.702           # of the experts' g * sigmoid(sharpness * g)


def _attention(m: Mapping[str, Any], where: str) -> dict:
    out = latent_attention_keys(m, where)
    if out.pop("scaling") is not None:
        raise ConfigError(f"config.json: '{where}rot.scaling' is not part of this design")
    window = None
    if m.get("mask") is not None:
        window = positive_int(section(m, "mask", where), "size", where + "mask.")
    return {**out, "window": window}


def _mamba2(m: Mapping[str, Any], where: str) -> dict:
    out = {k: positive_int(m, k, where)
           for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}
    if out["heads"] % out["groups"]:
        raise ConfigError(f"config.json: '{where}heads' ({out['heads']}) must be a multiple of "
                          f"'{where}groups' ({out['groups']})")
    if out["heads"] * out["vdim"] % out["norm_groups"]:
        raise ConfigError(f"config.json: '{where}norm_groups' ({out['norm_groups']}) must divide "
                          f"heads * vdim ({out['heads'] * out['vdim']})")
    return out


def _expert(data: Mapping[str, Any], key: str, where: str) -> tuple[int, float]:
    part = section(data, key, where)
    limit = number(part, "limit", f"{where}{key}.")
    if limit <= 0:
        raise ConfigError(f"config.json: '{where}{key}.limit' must be positive, got {limit}")
    return positive_int(part, "ff", f"{where}{key}."), limit


def _feed_forward(mlp: Any, where: str) -> "dict | None":
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping):
        raise ConfigError(f"config.json: '{where}mlp' must be an object or null")
    if mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: '{where}mlp.kind' is {mlp.get('kind')!r}; this design "
                          f"has 'moe'")
    where += "mlp."
    ff, limit = _expert(mlp, "expert", where)
    shared_ff, shared_limit = _expert(mlp, "shared", where)
    router = section(mlp, "router", where)
    where += "router."
    experts, top = positive_int(router, "experts", where), positive_int(router, "top", where)
    groups = section(router, "groups", where)
    count = positive_int(groups, "count", where + "groups.")
    keep = positive_int(groups, "keep", where + "groups.")
    if experts % count or keep > count:
        raise ConfigError(f"config.json: '{where}groups' cuts {experts} experts into {count} "
                          f"groups and keeps {keep}: the count must divide the experts and be at "
                          f"least what is kept")
    if top > experts // count * keep:
        raise ConfigError(f"config.json: '{where}top' ({top}) is more than the "
                          f"{experts // count * keep} experts of the kept groups")
    return {"ff": ff, "limit": limit, "shared_ff": shared_ff, "shared_limit": shared_limit,
            "experts": experts, "top": top, "groups": count, "keep": keep,
            "scale": number(router, "scale", where)}


_MIXERS = {"latent_attention": _attention, "mamba2": _mamba2}


@dataclass(frozen=True)
class PuripelConfig(ModelConfig):
    vocab: int
    model_width: int
    eps: float
    loop: "tuple[int, int, int] | None"      # (start, stop, times)
    # per layer: (mixer type, its parsed keys, the feed-forward's parsed keys or None), frozen
    layers: tuple

    # ------------------------------------------------------------------ parsing
    @staticmethod
    def from_json(data: Mapping[str, Any]) -> "PuripelConfig":
        width = positive("width", require(data, "width", int))
        eps = number(section(data, "norm", ""), "eps", "norm.")
        if eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        entries = data.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a nonempty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(entry, Mapping):
                raise ConfigError(f"config.json: 'layers[{i}]' must be an object")
            kind = entry.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: '{where}type' is {kind!r}; this design has "
                                  f"{sorted(_MIXERS)}")
            mixer = _MIXERS[kind](section(entry, "mixer", where), where + "mixer.")
            layers.append((kind, freeze(mixer), freeze(_feed_forward(entry.get("mlp"), where))))
        loop = None
        if data.get("loop") is not None:
            part = section(data, "loop", "")
            loop = tuple(part.get(k) for k in ("start", "stop", "times"))
            if (any(type(x) is not int for x in loop)
                    or not 0 <= loop[0] <= loop[1] <= len(layers) or loop[2] < 1):
                raise ConfigError("config.json: 'loop' needs integers 0 <= start <= stop <= the "
                                  "number of layers and times >= 1")
        return PuripelConfig(architecture=NAME,
                             vocab=positive("vocab", require(data, "vocab", int)),
                             model_width=width, eps=eps, loop=loop, layers=tuple(layers))

    def to_json(self) -> dict[str, Any]:
        layers = []
        for kind, mixer, mlp in self.layers:
            m = dict(mixer)
            if kind == "latent_attention":
                m["rot"] = {"base": m.pop("base"), "dims": m["rot_dim"]}
                window = m.pop("window")
                if window is not None:
                    m["mask"] = {"size": window}
            out_mlp = None
            if mlp is not None:
                f = dict(mlp)
                out_mlp = {"kind": "moe", "expert": {"ff": f["ff"], "limit": f["limit"]},
                           "shared": {"ff": f["shared_ff"], "limit": f["shared_limit"]},
                           "router": {"experts": f["experts"], "top": f["top"],
                                      "scale": f["scale"],
                                      "groups": {"count": f["groups"], "keep": f["keep"]}}}
            layers.append({"type": kind, "mixer": m, "mlp": out_mlp})
        out: dict[str, Any] = {"architecture": NAME, "vocab": self.vocab,
                               "width": self.model_width, "norm": {"eps": self.eps},
                               "layers": layers}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return json.loads(json.dumps(out))

    # ------------------------------------------------------------------ the model as data
    @property
    def width(self) -> int:
        return self.model_width

    @property
    def vocabulary(self) -> int:
        return self.vocab

    @property
    def max_positions(self) -> int:
        return MAX_POSITIONS

    @property
    def tied_output(self) -> bool:
        return True

    def _norm(self, tensor: str, kind: str = "rmsnorm") -> PartSpec:
        return PartSpec.of(kind, width=self.model_width, eps=self.eps, tensor=tensor)

    def _mixer(self, kind: str, m: dict) -> PartSpec:
        if kind == "mamba2":
            return PartSpec.of("mamba2", width=self.model_width, heads=m["heads"],
                               groups=m["groups"], state_dim=m["state"], value_dim=m["vdim"],
                               taps=m["conv"], norm_groups=m["norm_groups"], eps=self.eps)
        return PartSpec.of("latent_attention", width=self.model_width, heads=m["heads"],
                           key_dim=m["dim"], rotary_dim=m["rot_dim"], value_dim=m["vdim"],
                           q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=m["scale"],
                           theta=m["base"], eps=self.eps, window=m["window"], adjacent=True,
                           gated=False, exact_weights=True)

    def layer_specs(self) -> list[LayerSpec]:
        """A block with a norm before and after each sublayer: windowed latent attention or
        Mamba-2, then routed experts beside a shared one."""
        specs = []
        for i, (kind, mixer, mlp) in enumerate(self.layers):
            feed_forward, base = None, f"l{i}."
            after = {"mixer_after": self._norm("norm1b", "branch_rmsnorm")}
            if mlp is not None:
                f = dict(mlp)
                feed_forward = PartSpec.of(
                    "routed_experts", width=self.model_width, inner=f["ff"], experts=f["experts"],
                    top=f["top"], activation="clipped", gated=True, limit=f["limit"],
                    sharpness=GATE_SHARPNESS, scoring="grouped_sigmoid", bias_name="correction",
                    groups=f["groups"], keep=f["keep"], scale=f["scale"],
                    shared_inner=f["shared_ff"], shared_limit=f["shared_limit"])
                after["feed_forward_after"] = self._norm("norm2b", "branch_rmsnorm")
            specs.append(LayerSpec(
                block="sandwich", mixer=self._mixer(kind, dict(mixer)), feed_forward=feed_forward,
                norm=self._norm("norm1"), feed_forward_norm=self._norm("norm2"),
                prefixes=(("mixer", base + "mix."), ("feed_forward", base + "mlp."),
                          ("mixer_norm", base), ("feed_forward_norm", base),
                          ("mixer_after", base), ("feed_forward_after", base)),
                block_params=tuple(sorted(after.items()))))
        return specs

    def plan(self) -> list[PlanEntry]:
        """Layers in order, the looped ones ``times`` times in a row; every pass starts with its
        vector added to the stream."""
        n = len(self.layers)
        if self.loop is None:
            return [PlanEntry(i) for i in range(n)]
        start, stop, times = self.loop
        plan = [PlanEntry(i) for i in range(start)]
        for t in range(times):
            plan += [PlanEntry(i, adds_vector=t if i == start else None)
                     for i in range(start, stop)]
        return plan + [PlanEntry(i) for i in range(stop, n)]

    def plan_vectors(self) -> int:
        return self.loop[2] if self.loop is not None and self.loop[0] < self.loop[1] else 0

    def final_norm(self) -> PartSpec:
        return self._norm("norm")

    def tensor_names(self) -> dict[str, str]:
        return {"embedding": "embed", "final_norm": "final.", "output": "embed",
                "plan_vectors": "loop.step"}

    def unused_tensors(self) -> set[str]:
        """What a file may hold for a loop of no layers or a layer without a feed-forward."""
        out = {f"l{i}.{name}" for i, (_, _, mlp) in enumerate(self.layers) if mlp is None
               for name in ("norm2", "norm2b")}
        return out | ({"loop.step"} if self.plan_vectors() == 0 else set())

"""Typed configuration of the Sifasun decoder, read from its config.json.

The file names every size and every constant that differs between models of the design:

    {"architecture": "Sifasun", "vocab": V, "width": D, "norm": {"eps": e}, "logit_scale": s,
     "layers": [{"type": "attention" | "parallel", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F} | null,
                 "weights_of": j (optional)}, ...]}

* ``attention``: ``heads``, ``kv_heads``, ``dim`` (of a query or key head), ``vdim`` (the same: the
  values are the projected keys), ``scale``, ``mask.size`` (a window), ``rot`` (``base``, ``dims``,
  optional ``scaling.factor`` that divides the frequencies), ``softcap``.  q and k are divided by
  their root mean square per head; the softmax's denominator holds one more term, exp(0).
* ``parallel``: ``left`` (attention as above, with a weighted norm over the whole projection, no
  cap and an ordinary softmax), ``right`` (a gated linear recurrence: ``width``, ``blocks``, ``conv``
  taps), ``left_scale`` and ``right_scale``.
* ``weights_of``: the layer runs layer j's weights again (mixer, feed-forward and norms) with a
  cache or state of its own; the rest of its entry is layer j's.

A layer is x + norm1(mixer(x)), then x + norm2(mlp(x)), the norms' weights stored around zero; the
output matrix is the embedding table, its logits times ``logit_scale``.  Layer i's tensors are named
``l<i>.*``.  A model of this design has no position limit of its own.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from typing import Any, Mapping

from .model import (ConfigError, LayerSpec, ModelConfig, PartSpec, PlanEntry, positive, require,
                    number as _number, positive_int as _int, section as _section)

NAME = "Sifasun"
MAX_POSITIONS = 1 << 20          # the design names none
KINDS = ("attention", "parallel")
ATTENTION_KEYS = {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"}


def _freeze(value):
    if isinstance(value, dict):
        return tuple(sorted((k, _freeze(v)) for k, v in value.items()))
    return value


def _unknown(m: Mapping[str, Any], allowed: "set[str]", where: str) -> None:
    unknown = {k for k in set(m) - allowed if m[k] is not None and m[k] is not False}
    if unknown:
        raise ConfigError(f"config.json: '{where}' has keys this design does not know: "
                          f"{sorted(unknown)}")


def _rotation(m: Mapping[str, Any], where: str, dim: int) -> "dict | None":
    if m.get("rot") is None:
        return None
    rot, at = _section(m, "rot", where), where + "rot."
    dims = rot.get("dims")
    if type(dims) is not int or dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"config.json: '{at}dims' ({dims!r}) must be an even number from 0 to "
                          f"'{where}dim' ({dim})")
    base = _number(rot, "base", at)
    if base <= 0:
        raise ConfigError(f"config.json: '{at}base' must be positive")
    factor = None
    if rot.get("scaling") is not None:
        factor = _number(_section(rot, "scaling", at), "factor", at + "scaling.")
        if factor <= 0:
            raise ConfigError(f"config.json: '{at}scaling.factor' must be positive")
    _unknown(rot, {"dims", "base", "scaling"}, at)
    return {"base": base, "dims": dims, "factor": factor}


def _attention(m: Mapping[str, Any], where: str, capped: bool) -> dict:
    heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: '{where}heads' ({heads}) must be a multiple of "
                          f"'{where}kv_heads' ({kv_heads})")
    dim, vdim = _int(m, "dim", where), _int(m, "vdim", where)
    if dim != vdim:
        raise ConfigError(f"config.json: '{where}vdim' ({vdim}) must be '{where}dim' ({dim}): the "
                          f"values are the projected keys")
    window = None
    if m.get("mask") is not None:
        window = _int(_section(m, "mask", where), "size", where + "mask.")
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "scale": _number(m, "scale", where),
           "window": window, "rot": _rotation(m, where, dim)}
    if capped:
        out["softcap"] = None
        if m.get("softcap") is not None:
            out["softcap"] = _number(m, "softcap", where)
            if out["softcap"] <= 0:
                raise ConfigError(f"config.json: '{where}softcap' must be positive")
    _unknown(m, ATTENTION_KEYS | ({"softcap"} if capped else set()), where)
    return out


def _recurrence(m: Mapping[str, Any], where: str) -> dict:
    width, blocks = _int(m, "width", where), _int(m, "blocks", where)
    if width % blocks:
        raise ConfigError(f"config.json: '{where}blocks' ({blocks}) must divide '{where}width' "
                          f"({width})")
    _unknown(m, {"width", "blocks", "conv"}, where)
    return {"width": width, "blocks": blocks, "conv": _int(m, "conv", where)}


def _mixer(kind: str, m: Mapping[str, Any], where: str) -> dict:
    if kind == "attention":
        return _attention(m, where, capped=True)
    _unknown(m, {"left", "right", "left_scale", "right_scale"}, where)
    return {"left": _attention(_section(m, "left", where), where + "left.", capped=False),
            "right": _recurrence(_section(m, "right", where), where + "right."),
            "left_scale": _number(m, "left_scale", where),
            "right_scale": _number(m, "right_scale", where)}


def _feed_forward(mlp: Any, where: str) -> "int | None":
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping):
        raise ConfigError(f"config.json: '{where}mlp' must be an object or null")
    if mlp.get("kind") != "dense":
        raise ConfigError(f"config.json: '{where}mlp.kind' is {mlp.get('kind')!r}; this design has "
                          f"'dense'")
    _unknown(mlp, {"kind", "ff"}, where + "mlp.")
    return _int(mlp, "ff", where + "mlp.")


@dataclass(frozen=True)
class SifasunConfig(ModelConfig):
    vocab: int
    model_width: int
    eps: float
    output_scale: float
    # per layer: (type, the mixer's parsed keys, frozen, the feed-forward's size or None)
    layers: tuple
    # per layer: the layer whose weights it runs (its own index: it has tensors of its own)
    weights: tuple

    # ------------------------------------------------------------------ parsing
    @staticmethod
    def from_json(data: Mapping[str, Any]) -> "SifasunConfig":
        eps = _number(_section(data, "norm", ""), "eps", "norm.")
        if eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        entries = data.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a nonempty list")
        layers, named = [], []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(entry, Mapping):
                raise ConfigError(f"config.json: 'layers[{i}]' must be an object")
            kind = entry.get("type")
            if kind not in KINDS:
                raise ConfigError(f"config.json: '{where}type' is {kind!r}; this design has "
                                  f"{' and '.join(repr(k) for k in KINDS)}")
            mixer = _mixer(kind, _section(entry, "mixer", where), where + "mixer.")
            layers.append((kind, _freeze(mixer), _feed_forward(entry.get("mlp"), where)))
            named.append(entry.get("weights_of"))
        weights = []
        for i, j in enumerate(named):
            at, seen = i, {i}
            while named[at] is not None:       # (a layer may name one that names another)
                j = named[at]
                if type(j) is not int or not 0 <= j < len(layers) or j in seen:
                    raise ConfigError(f"config.json: 'layers[{at}].weights_of' is {j!r}: it must "
                                      f"lead to a layer that has tensors of its own")
                seen.add(j)
                at = j
            if layers[at] != layers[i]:
                raise ConfigError(f"config.json: 'layers[{i}]' uses the weights of layer {at} but "
                                  f"its entry is not that layer's")
            weights.append(at)
        scale = data.get("logit_scale")
        return SifasunConfig(architecture=NAME,
                             vocab=positive("vocab", require(data, "vocab", int)),
                             model_width=positive("width", require(data, "width", int)), eps=eps,
                             output_scale=1.0 if scale is None else _number(data, "logit_scale", ""),
                             layers=tuple(layers), weights=tuple(weights))

    def to_json(self) -> dict[str, Any]:
        def attention(a: dict) -> dict:
            out: dict[str, Any] = {"heads": a["heads"], "kv_heads": a["kv_heads"], "dim": a["dim"],
                                   "vdim": a["dim"], "scale": a["scale"]}
            if a["window"] is not None:
                out["mask"] = {"size": a["window"]}
            if a["rot"] is not None:
                rot = dict(a["rot"])
                out["rot"] = {"base": rot["base"], "dims": rot["dims"]}
                if rot["factor"] is not None:
                    out["rot"]["scaling"] = {"factor": rot["factor"]}
            if a.get("softcap") is not None:
                out["softcap"] = a["softcap"]
            return out

        layers = []
        for i, (kind, mixer, ff) in enumerate(self.layers):
            m = dict(mixer)
            if kind == "attention":
                out_mixer = attention(m)
            else:
                out_mixer = {"left": attention(dict(m["left"])), "right": dict(m["right"]),
                             "left_scale": m["left_scale"], "right_scale": m["right_scale"]}
            entry = {"type": kind, "mixer": out_mixer,
                     "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
            if self.weights[i] != i:
                entry["weights_of"] = self.weights[i]
            layers.append(entry)
        out = {"architecture": NAME, "vocab": self.vocab, "width": self.model_width,
               "norm": {"eps": self.eps}, "logit_scale": self.output_scale, "layers": layers}
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

    def _norm(self, kind: str, tensor: str, gain: float = 1.0) -> PartSpec:
        return PartSpec.of(kind, width=self.model_width, eps=self.eps, tensor=tensor, offset=1.0,
                           gain=gain)

    def _attention_part(self, a: dict, **more) -> PartSpec:
        rot = dict(a["rot"]) if a["rot"] is not None else None
        return PartSpec.of("sink_attention", width=self.model_width, heads=a["heads"],
                           kv_heads=a["kv_heads"], key_dim=a["dim"], value_dim=a["dim"],
                           scale=a["scale"], eps=self.eps, values_from_keys=True, adjacent=False,
                           window=a["window"], rotary_dim=rot["dims"] if rot else 0,
                           theta=rot["base"] if rot else 10000.0,
                           frequency_factor=rot["factor"] if rot else None, **more)

    def _mixer_part(self, kind: str, m: dict) -> PartSpec:
        if kind == "attention":
            # a turn keeps a head's length, so the norm without a weight may stand before it
            return self._attention_part(m, norm="head", norm_weighted=False,
                                        softcap=m["softcap"], sink="zero")
        right = dict(m["right"])
        return PartSpec.of(
            "parallel", width=self.model_width, eps=self.eps, combine="joined_sum",
            scales=(m["left_scale"], m["right_scale"]),
            branches=(("left", self._attention_part(dict(m["left"]), norm="whole", sink=None)),
                      ("right", PartSpec.of("gated_recurrence", width=self.model_width,
                                            inner=right["width"], blocks=right["blocks"],
                                            taps=right["conv"]))))

    def _own(self) -> "list[int]":
        """The layers that have tensors of their own, in order."""
        return [i for i, j in enumerate(self.weights) if i == j]

    def layer_specs(self) -> list[LayerSpec]:
        specs = []
        for i in self._own():
            kind, mixer, ff = self.layers[i]
            base = f"l{i}."
            feed_forward = None
            if ff is not None:
                feed_forward = PartSpec.of("gated_mlp", width=self.model_width, inner=ff,
                                           activation="silu", names=("gate", "up", "down"))
            specs.append(LayerSpec(
                block="sublayer_norm", mixer=self._mixer_part(kind, dict(mixer)),
                feed_forward=feed_forward, norm=self._norm("branch_rmsnorm", "norm1"),
                feed_forward_norm=self._norm("branch_rmsnorm", "norm2"),
                prefixes=(("mixer", base + "mix."), ("feed_forward", base + "mlp."),
                          ("mixer_norm", base), ("feed_forward_norm", base))))
        return specs

    def plan(self) -> list[PlanEntry]:
        at = {i: k for k, i in enumerate(self._own())}
        return [PlanEntry(at[j]) for j in self.weights]

    def final_norm(self) -> PartSpec:
        # the logits' scale rides on the final norm's weight
        return self._norm("rmsnorm", "norm", gain=self.output_scale)

    def unused_tensors(self) -> set[str]:
        """The second sublayer's norm of a layer without a feed-forward, which a weight file of
        this design may hold."""
        return {f"l{i}.norm2" for i in self._own() if self.layers[i][2] is None}

    def tensor_names(self) -> dict[str, str]:
        return {"embedding": "embed", "final_norm": "final.", "output": "embed"}

"""The Sifasun configuration: parsing, the layer specs and plan it gives the generic decoder, the
tensors it expects, what every layer run keeps, and the errors that name the key."""

import copy

import pytest
import torch

import plain_sifasun as ps
import sifasun_configs as sc
from distengine_b200.config import ConfigError
from distengine_b200.config.sifasun import SifasunConfig
from distengine_b200.models import expected_tensors
from distengine_b200.registry import resolve


@pytest.mark.parametrize("name", sorted(sc.ALL))
def test_round_trip_and_tensors(name):
    architecture, config = resolve(sc.ALL[name])
    assert architecture.name == "Sifasun" and isinstance(config, SifasunConfig)
    assert config.to_json() == sc.ALL[name]
    assert SifasunConfig.from_json(config.to_json()) == config
    expected, vectors, optional = expected_tensors(config)
    assert {k: tuple(v) for k, v in expected.items()} == ps.tensor_shapes(sc.ALL[name])
    assert not optional and config.tied_output
    # norms whose weight is stored around zero are not drawn around one
    assert "final.norm" not in vectors and "l0.norm1" not in vectors


def test_layers_that_use_another_layers_weights_run_again():
    config = SifasunConfig.from_json(sc.SIF_A)
    assert len(config.layer_specs()) == 3
    assert [e.layer for e in config.plan()] == [0, 1, 2, 0, 1, 0]
    assert all(e.reads_cache_of is None for e in config.plan())
    assert not any(name.startswith(("l3.", "l4.", "l5.")) for name in expected_tensors(config)[0])
    chain = copy.deepcopy(sc.SIF_A)                # a layer that names one that names another
    chain["layers"][5]["weights_of"] = 3
    assert SifasunConfig.from_json(chain).plan() == config.plan()
    later = sc.model(8, 9, [sc.layer(sc.attention(1, 1, 4, 1.0, 3), 5, 1),
                            sc.layer(sc.attention(1, 1, 4, 1.0, 3), 5)])
    parsed = SifasunConfig.from_json(later)
    assert [e.layer for e in parsed.plan()] == [0, 0]
    assert "l1.mix.q" in expected_tensors(parsed)[0] and "l0.mix.q" not in expected_tensors(parsed)[0]


def test_layer_specs_name_the_parts():
    specs = SifasunConfig.from_json(sc.SIF_A).layer_specs()
    assert [s.block for s in specs] == ["sublayer_norm"] * 3
    assert [s.mixer.kind for s in specs] == ["sink_attention", "parallel", "sink_attention"]
    assert [s.feed_forward is None for s in specs] == [False, False, True]
    first = specs[0].mixer.params
    assert (first["window"], first["softcap"], first["sink"]) == (5, 3.0, "zero")
    assert (first["norm"], first["norm_weighted"], first["frequency_factor"]) == ("head", False, 2.5)
    assert first["values_from_keys"] and not first["adjacent"]
    beside = specs[1].mixer.params
    assert beside["combine"] == "joined_sum" and beside["scales"] == (0.7, 1.2)
    left, right = beside["branches"][0][1].params, beside["branches"][1][1].params
    assert (left["norm"], left["sink"], left["window"]) == ("whole", None, 21)
    assert left["frequency_factor"] is None and "softcap" not in left
    assert (right["inner"], right["blocks"], right["taps"]) == (15, 3, 4)
    norm = SifasunConfig.from_json(sc.SIF_A).final_norm().params
    assert (norm["offset"], norm["gain"]) == (1.0, 0.7)


def test_what_every_layer_run_keeps():
    from distengine_b200.models.decoder import DecoderModel
    model = DecoderModel(SifasunConfig.from_json(sc.SIF_A), torch.float32, "meta")
    specs = model.cache_specs()
    assert len(specs) == 6 and all(s is not None for s in specs)
    assert specs[0] == specs[3] == specs[5] and specs[0].window == 5 and specs[0].v_dim == 10
    pages, state = specs[1]
    assert pages.window == 21 and pages.head_dim == pages.v_dim == 7
    # the state, then a ring of one row a tap, both on multiples of four floats
    assert state.shape == (16 + 4 * 15,) and state.dtype == torch.float32
    one_tap = DecoderModel(SifasunConfig.from_json(sc.SIF_B), torch.float32, "meta").cache_specs()
    assert one_tap[2][1].shape == (64,)
    assert DecoderModel(SifasunConfig.from_json(sc.SIF_C), torch.float32,
                        "meta").cache_specs()[2].window is None


def test_a_layer_without_feed_forward_may_have_its_norm():
    assert SifasunConfig.from_json(sc.SIF_A).unused_tensors() == {"l2.norm2"}


@pytest.mark.parametrize("change, key", [
    (lambda c: c["layers"][0].update(type="mamba2"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "layers[0].mixer.heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=9), "layers[0].mixer.vdim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "layers[0].mixer.rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "layers[0].mixer.rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "scaling.factor"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("factor"), "scaling.factor"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "layers[0].mixer.mask.size"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "layers[0].mixer.softcap"),
    (lambda c: c["layers"][0]["mixer"].update(sinks=2), "sinks"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(softcap=2.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(blocks=4), "right.blocks"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "right.conv"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "layers[1].mlp.kind"),
    (lambda c: c["layers"][3].update(weights_of=6), "layers[3].weights_of"),
    (lambda c: c["layers"][0].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=1), "layers[3]"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
])
def test_errors_name_the_key(change, key):
    config = copy.deepcopy(sc.SIF_A)
    change(config)
    with pytest.raises(ConfigError) as error:
        SifasunConfig.from_json(config)
    assert key in str(error.value)

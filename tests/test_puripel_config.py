"""The Puripel configuration: parsing, the layer specs and plan it gives the generic decoder, the
tensors it expects, what every layer run keeps, and the errors that name the key."""

import copy

import pytest
import torch

import plain_puripel as pp
import puripel_configs as pc
from distengine_b200.config import ConfigError
from distengine_b200.config.puripel import PuripelConfig
from distengine_b200.models import expected_tensors
from distengine_b200.registry import resolve


@pytest.mark.parametrize("name", sorted(pc.ALL))
def test_round_trip_and_tensors(name):
    architecture, config = resolve(pc.ALL[name])
    assert architecture.name == "Puripel" and isinstance(config, PuripelConfig)
    assert config.to_json() == pc.ALL[name]
    assert PuripelConfig.from_json(config.to_json()) == config
    expected, vectors, optional = expected_tensors(config)
    assert {k: tuple(v) for k, v in expected.items()} == pp.tensor_shapes(pc.ALL[name])
    assert {"final.norm", "l0.norm1", "l0.norm1b"} <= vectors and not optional
    assert config.tied_output


def test_every_pass_of_the_loop_starts_with_its_vector():
    config = PuripelConfig.from_json(pc.PUR_A)
    plan = [(e.layer, e.adds_vector) for e in config.plan()]
    assert plan == pp.run_order(pc.PUR_A)
    assert plan == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert config.plan_vectors() == 3
    once = copy.deepcopy(pc.PUR_A)
    once["loop"]["times"] = 1                      # a single pass has its vector too
    config = PuripelConfig.from_json(once)
    assert [e.adds_vector for e in config.plan()] == [None, 0, None, None]
    assert expected_tensors(config)[0]["loop.step"] == (1, 42)
    none = copy.deepcopy(pc.PUR_A)
    none["loop"].update(start=2, stop=2)           # a loop of no layers
    config = PuripelConfig.from_json(none)
    assert [(e.layer, e.adds_vector) for e in config.plan()] == [(i, None) for i in range(4)]
    assert "loop.step" not in expected_tensors(config)[0]
    assert "loop.step" in config.unused_tensors()
    assert PuripelConfig.from_json(pc.PUR_B).plan_vectors() == 0


def test_layer_specs_name_the_parts():
    specs = PuripelConfig.from_json(pc.PUR_A).layer_specs()
    assert [s.block for s in specs] == ["sandwich"] * 4
    assert [s.mixer.kind for s in specs] == ["mamba2", "latent_attention"] * 2
    assert [s.feed_forward is None for s in specs] == [False, True, False, False]
    assert specs[3].mixer.params["window"] == 21 and specs[1].mixer.params["window"] == 5
    assert specs[1].mixer.params["adjacent"] and not specs[1].mixer.params["gated"]
    experts = specs[0].feed_forward.params
    assert (experts["groups"], experts["keep"], experts["scale"]) == (3, 2, 1.7)
    assert (experts["limit"], experts["shared_limit"], experts["shared_inner"]) == (0.8, 0.6, 13)
    assert dict(specs[1].block_params).keys() == {"mixer_after"}


def test_what_every_layer_run_keeps():
    from distengine_b200.models.decoder import DecoderModel
    model = DecoderModel(PuripelConfig.from_json(pc.PUR_A), torch.float32, "meta")
    specs = model.cache_specs()
    assert len(specs) == 8 and all(s is not None for s in specs)
    assert specs[1] == specs[3] == specs[5] and specs[1].window == 5
    assert specs[1].values_in_keys and specs[1].head_dim == 9 and specs[1].v_dim == 7
    assert specs[7].window == 21
    # state rows, then the convolution's kept inputs, both on multiples of four floats
    assert specs[0].shape == (92 + 3 * (18 + 2 * 3 * 5),) and specs[0].dtype == torch.float32
    assert specs[2] == specs[4] and specs[2].shape == (316,)


def test_a_window_is_optional_and_a_layer_without_feed_forward_may_have_its_norms():
    config = copy.deepcopy(pc.PUR_B)
    del config["layers"][0]["mixer"]["mask"]
    parsed = PuripelConfig.from_json(config)
    assert parsed.layer_specs()[0].mixer.params["window"] is None
    assert parsed.to_json() == config
    assert {"l2.norm2", "l2.norm2b"} <= parsed.unused_tensors()


@pytest.mark.parametrize("change, key", [
    (lambda c: c["layers"][0].update(type="attention"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "layers[0].mixer.heads"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=4), "layers[0].mixer.norm_groups"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "layers[0].mixer.conv"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=5), "layers[1].mixer.rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), "layers[1].mixer.rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "layers[1].mixer.mask.size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(
        scaling={"factor": 2, "original": 8, "fast": 2, "slow": 1}), "rot.scaling"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "layers[0].mlp.kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "layers[0].mlp.router.top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "router.groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "router.groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "layers[0].mlp.router.scale"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "layers[0].mlp.expert.limit"),
    (lambda c: c["layers"][0]["mlp"].pop("shared"), "shared"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
])
def test_errors_name_the_key(change, key):
    config = copy.deepcopy(pc.PUR_A)
    change(config)
    with pytest.raises(ConfigError) as error:
        PuripelConfig.from_json(config)
    assert key in str(error.value)

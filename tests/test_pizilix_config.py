"""The Pizilix configuration: reading, refusing, writing back, and the parts its model is
assembled from.  No GPU."""
from __future__ import annotations

import copy

import pytest

from helix_runtime_b200.config import ConfigError, architecture_for
from helix_runtime_b200.config.pizilix import PizilixConfig
from helix_runtime_b200.models import DecoderModel
from pizilix_configs import CONFIGS, tensors_for


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip_and_registry(name):
    document = CONFIGS[name]
    entry = architecture_for(document)
    assert entry.name == "Pizilix"
    config = entry.config_from_dict(document)
    assert PizilixConfig.from_dict(config.to_dict()) == config
    spec = entry.build_spec(config)
    assert all(block.arrangement == "pre_norm" for block in spec.blocks)
    for block, layer in zip(spec.blocks, document["layers"]):
        assert (block.feed_forward is None) == (layer["mlp"] is None)
    assert spec.lm_head.get("softcap") == document.get("logit_softcap")
    assert spec.lm_head.tensors["weight"] == spec.embedding.tensors["weight"] == "embed"


def test_the_order_of_layers_and_where_the_input_joins_again():
    entry = architecture_for(CONFIGS["mixed"])
    spec = entry.build_spec(entry.config_from_dict(CONFIGS["mixed"]))
    assert [run.block for run in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [run.add_embedding for run in spec.schedule] == [False, False, False, True, False, True,
                                                            False, False]
    document = copy.deepcopy(CONFIGS["mixed"])
    document["loop"] = {"start": 0, "stop": 4, "times": 1}
    spec = entry.build_spec(entry.config_from_dict(document))
    assert [run.block for run in spec.schedule] == [0, 1, 2, 3]
    assert not any(run.add_embedding for run in spec.schedule)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_model_binds_exactly_the_checkpoint_tensors(name):
    import torch
    document = CONFIGS[name]
    entry = architecture_for(document)
    tensors = tensors_for(document, 1, torch.float32)
    model = DecoderModel(entry.build_spec(entry.config_from_dict(document)))
    requests = {request.name: tuple(request.shape) for request in model.tensor_requests()}
    assert requests == {key: tuple(value.shape) for key, value in tensors.items()}
    kv, state = model.cache_needs()
    for index, run in enumerate(model.schedule):        # every run owns its cache or state
        layer = document["layers"][run.block]
        mixer = layer["mixer"]
        if layer["type"] == "attention":
            assert index not in state
            assert kv[index].window is None
            assert kv[index].chunk == (mixer.get("mask") or {}).get("size")
            assert kv[index].kv_heads == mixer["kv_heads"] and kv[index].head_dim >= mixer["dim"]
        else:
            assert index not in kv
            assert state[index].shape == (mixer["conv"] * mixer["width"],)
            assert state[index].dtype == torch.float32


def test_optional_keys_may_be_left_out():
    document = copy.deepcopy(CONFIGS["plain"])
    config = PizilixConfig.from_dict(document)
    assert config.logit_softcap is None and config.loop is None
    attention = config.layers[0].mixer
    assert attention.softcap is None and attention.chunk is None and attention.scaling is None
    for key in ("kv_heads", "vdim"):
        del document["layers"][0]["mixer"][key]
    del document["layers"][0]["mixer"]["rot"]["dims"]
    relaxed = PizilixConfig.from_dict(document).layers[0].mixer
    assert relaxed.kv_heads == relaxed.heads and relaxed.rot_dims == relaxed.dim


@pytest.mark.parametrize("change,complaint", [
    (lambda d: d["layers"][0].update(type="conv"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(blocks=7), "blocks"),
    (lambda d: d["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][0]["mixer"].pop("width"), "width"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=16), "vdim"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda d: d["layers"][1]["mixer"].update(softcap=-2.0), "softcap"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(base=1.0), "rot.base"),
    (lambda d: d["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d.update(loop={"start": 2, "stop": 9, "times": 2}), "loop"),
    (lambda d: d.update(loop={"start": 1, "stop": 3, "times": 0}), "loop"),
    (lambda d: d.update(logit_softcap=0.0), "logit_softcap"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_what_the_configuration_refuses(change, complaint):
    document = copy.deepcopy(CONFIGS["mixed"])
    change(document)
    with pytest.raises(ConfigError, match=complaint):
        PizilixConfig.from_dict(document)


@pytest.mark.parametrize("dims,base,scaling", [
    (20, 30000.0, (5.0, 640, 16.0, 2.0)), (12, 10000.0, (4.0, 24, 8.0, 1.0)),
    (4, 77.0, (3.0, 10, 2.0, 0.25)), (64, 10000.0, None), (2, 5.0, (8.0, 4, 1.0, 0.5))])
def test_rotary_table(dims, base, scaling):
    """The table of a position encoding holds the plain frequencies' cosines and sines times the
    amplitude, and two encodings with the same numbers hold one table."""
    import numpy as np
    import torch

    import plain_pizilix as plain
    from helix_runtime_b200.config.spec import PartSpec
    from helix_runtime_b200.parts.base import build_part
    keys = ("factor", "original", "fast", "slow")
    params = {"theta": base, "exact_theta": True, "head_dim": dims + 6, "rotary_dim": dims,
              "max_positions": 300}
    if scaling is not None:
        params["scaling"] = dict(zip(keys, scaling))
    parts = [build_part("position", PartSpec("rotary", params), 32) for _ in range(2)]
    for part in parts:
        part.bind({}, torch.float32, torch.device("cpu"))
    assert parts[0].cos is parts[1].cos
    frequencies, amplitude = plain.rotary_frequencies(dims, base,
                                                      None if scaling is None else dict(zip(keys, scaling)))
    angle = np.arange(300)[:, None] * frequencies[None, :]
    np.testing.assert_allclose(parts[0].cos.numpy(), np.cos(angle) * amplitude, rtol=0, atol=2e-7)
    np.testing.assert_allclose(parts[0].sin.numpy(), np.sin(angle) * amplitude, rtol=0, atol=2e-7)


def test_parts_that_do_not_fit_are_refused():
    from helix_runtime_b200.config.spec import PartSpec
    from helix_runtime_b200.parts.base import build_part
    rotary = PartSpec("rotary", {"theta": 100.0, "head_dim": 16, "max_positions": 64})
    base = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "values": "keys", "position": rotary}
    names = {name: name for name in ("q", "k", "o")}
    build_part("mixer", PartSpec("paged_attention", base, names), 32)
    for change in ({"values": "queries"}, {"value_dim": 8}, {"short_conv": 3},
                   {"output_gate": "sigmoid"}, {"softcap": -1.0},
                   {"position": PartSpec("none", {"head_dim": 16})}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("paged_attention", {**base, **change}, names), 32)
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("gated_recurrence", {"width": 10, "blocks": 3}, {}), 32)

"""The Manatar configuration: reading, refusing, writing back, and the parts its model is
assembled from; the plain implementation's mechanisms against each other.  No GPU."""
from __future__ import annotations

import copy

import numpy as np
import pytest

import plain_manatar as plain
from helix_runtime_b200.config import ConfigError, architecture_for
from helix_runtime_b200.config.manatar import ManatarConfig
from helix_runtime_b200.models import DecoderModel
from helix_runtime_b200.models.decoder import EMBEDDING_STATE
from manatar_configs import CONFIGS, tensors_for


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip_and_registry(name):
    document = CONFIGS[name]
    entry = architecture_for(document)
    assert entry.name == "Manatar"
    config = entry.config_from_dict(document)
    assert ManatarConfig.from_dict(config.to_dict()) == config
    spec = entry.build_spec(config)
    assert all(block.arrangement == "output_norm" and block.mixer_norm is None for block in spec.blocks)
    for block, run, layer in zip(spec.blocks, spec.schedule, document["layers"]):
        assert (block.feed_forward is None) == (layer["mlp"] is None)
        assert run.cache_from == layer["mixer"].get("kv_from")
        assert block.mixer_connection["scale"] == document["residual_mult"]
    pairs = document.get("embedding", {}).get("bigram")
    assert spec.embedding.get("pairs") == pairs and ("pairs" in spec.embedding.tensors) == bool(pairs)


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
    assert (EMBEDDING_STATE in state) == ("embedding" in document)
    for index, layer in enumerate(document["layers"]):
        mixer = layer["mixer"]
        if layer["type"] == "mlstm":
            assert index not in kv and state[index].dtype == torch.float32
            floats = mixer["heads"] * (mixer["dim"] * (mixer["vdim"] + 1) + 1)
            assert state[index].shape[0] >= floats
            continue
        # a layer that uses another's keys has no pages, but keeps its own filter's inputs
        shares = mixer.get("kv_from") is not None
        assert (index in kv) == (not shares)
        if not shares:
            assert kv[index].kv_heads == mixer["kv_heads"]
            assert kv[index].head_dim >= max(2 * mixer["dim"], mixer["vdim"])
        channels = mixer["heads"] * 2 * mixer["dim"]
        if not shares:
            channels += mixer["kv_heads"] * (2 * mixer["dim"] + mixer["vdim"])
        size = (mixer["conv"] - 1) * channels
        if size:
            assert state[index].shape == (size + size % 2,) and state[index].dtype == torch.float32
        else:
            assert index not in state


def test_optional_keys_may_be_left_out():
    document = copy.deepcopy(CONFIGS["plain"])
    config = ManatarConfig.from_dict(document)
    assert config.pairs is None and config.layers[0].mixer.scaling is None
    assert config.layers[0].mixer.kv_from is None
    for key in ("kv_heads", "vdim", "conv"):
        del document["layers"][0]["mixer"][key]
    del document["layers"][0]["mixer"]["rot"]["dims"]
    del document["layers"][1]["mixer"]["vdim"]
    del document["layers"][0]["mlp"]["shared"]
    relaxed = ManatarConfig.from_dict(document).layers
    assert relaxed[0].mixer.kv_heads == relaxed[0].mixer.heads
    assert relaxed[0].mixer.rot_dims == relaxed[0].mixer.vdim == relaxed[0].mixer.dim
    assert relaxed[0].mixer.conv == 1 and relaxed[1].mixer.vdim == relaxed[1].mixer.dim
    assert relaxed[0].mlp.shared_ff == 0


@pytest.mark.parametrize("change,complaint", [
    (lambda d: d["layers"][0].update(type="rglru"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda d: d["layers"][1]["mixer"].update(kv_from=1), "kv_from"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda d: d["layers"][1]["mixer"].update(dim=20, rot={"base": 10.0, "dims": 4}), "another shape"),
    (lambda d: d["layers"][2]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][3]["mlp"]["router"].update(top=6), "router.top"),
    (lambda d: d["layers"][3]["mlp"].update(kind="dense9"), "kind"),
    (lambda d: d["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda d: d["embedding"]["bigram"].update(mul_prev=1.5), "mul_prev"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_refusals(change, complaint):
    document = copy.deepcopy(CONFIGS["mixed"])
    change(document)
    with pytest.raises(ConfigError, match=complaint):
        ManatarConfig.from_dict(document)


def test_the_shared_row_carries_both_maps():
    """Scores of a map from the joined key row and a query row that is zero outside its part are
    the map's own: how the engine caches and reads two maps."""
    rng = np.random.default_rng(3)
    q, k, v = rng.normal(size=(9, 2, 6)), rng.normal(size=(9, 2, 6)), rng.normal(size=(9, 5))
    joined = k.reshape(9, 12)
    for part in (0, 1):
        row = np.zeros((9, 12))
        row[:, 6 * part:6 * part + 6] = q[:, part]
        np.testing.assert_allclose(plain.causal_softmax_map(row, joined, v, 0.3),
                                   plain.causal_softmax_map(q[:, part], k[:, part], v, 0.3), atol=1e-12)


def test_the_running_maximum_is_a_change_of_scale():
    """The matrix memory against its closed form without a running maximum: weights of all earlier
    tokens, the divisor's bound and its small constant in the same scale."""
    rng = np.random.default_rng(4)
    length, dim, vdim = 40, 5, 3
    q, k, v = (rng.normal(size=(length, n)) for n in (dim, dim, vdim))
    log_in, log_forget = plain.lstm_gates(4.0 * rng.normal(size=length), 3.0 + 3.0 * rng.normal(size=length), 9.0)
    got = plain.matrix_lstm(q, k, v, log_in, log_forget)
    total = np.cumsum(log_forget)
    for t in range(length):
        log_weights = log_in[:t + 1] + total[t] - total[:t + 1]
        m = max(total[t], log_weights.max())
        m = max([total[t]] + [log_in[s] + total[t] - total[s] for s in range(t + 1)])
        weights = np.exp(log_weights - m) * (k[:t + 1] @ q[t])
        want = weights @ v[:t + 1] / (max(abs(weights.sum()), np.exp(-m)) + 1e-6)
        np.testing.assert_allclose(got[t], want, atol=1e-9)

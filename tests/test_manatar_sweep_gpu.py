"""Randomly drawn Manatar configurations through the engine against the plain implementation: the
order and number of layers, layers that use an earlier layer's keys and values, every size of the
two mixers (heads, grouped key/value heads, maps of 4 to 136 coordinates, values of 6 to 264,
filters of 1 to 6 taps, rotation of some or all coordinates with and without stretched
frequencies; matrices of 4 to 320 by 7 to 264), dense and routed feed-forwards or none, with and
without a shared expert and a table of pairs (a head of one or two numbers is normed to little more
than their signs, which anything that rounds differently turns where they are near zero: no model
has such heads); every model is replayed as mixed batches over a pool
made for its live requests only."""
from __future__ import annotations

import math
import os

import numpy as np
import pytest
import torch

import traces
from conftest import random_tokens
from engine_harness import Harness
from helix_runtime_b200.weights.random_init import write_model_folder
from manatar_configs import tensors_for
from plain_manatar import PlainManatar
from test_manatar_model_gpu import Expected, check_rows

pytestmark = pytest.mark.gpu


def draw_config(seed: int):
    rng = np.random.default_rng(9000 + seed)
    pick = lambda values: values[int(rng.integers(0, len(values)))]
    width = pick([40, 64, 72, 100, 128, 136, 256])
    layers = []
    for index in range(int(rng.integers(1, 6))):
        sources = [i for i, layer in enumerate(layers)
                   if layer["type"] == "attention" and "kv_from" not in layer["mixer"]]
        if rng.random() < 0.6:
            kind = "attention"
            if sources and rng.random() < 0.4:
                source = pick(sources)
                mixer = dict(layers[source]["mixer"], kv_from=source, conv=pick([1, 2, 3, 4, 6]),
                             diff=pick([0.1, 0.5, 0.8]))
                mixer["scale"] = pick([1.0, 2.0, 4.0]) / math.sqrt(mixer["dim"])
            else:
                dim, kv_heads = pick([4, 6, 9, 16, 20, 32, 48, 64, 72, 136]), pick([1, 1, 2, 3])
                vdim = pick([6, 7, 16, max(2 * dim, 6), 2 * dim + 6, max(dim, 6), 40, 128]) if rng.random() < 0.9 else 264
                rot = {"base": float(pick([100.0, 10000.0, 500000.0])),
                       "dims": pick([d for d in (2, dim // 4 * 2, dim) if d % 2 == 0 and d > 0])}
                if rng.random() < 0.6:
                    rot["scaling"] = {"factor": float(pick([1.5, 4.0, 40.0])),
                                      "original": pick([8, 32, 64, 512]),
                                      "fast": float(pick([1.0, 4.0, 32.0])),
                                      "slow": float(pick([0.25, 1.0, 2.0]))}
                mixer = {"heads": kv_heads * pick([1, 2, 3, 4]), "kv_heads": kv_heads, "dim": dim,
                         "vdim": vdim, "scale": pick([1.0, 2.0, 4.0]) / math.sqrt(dim),
                         "conv": pick([1, 2, 3, 4, 4, 6]), "diff": pick([0.1, 0.3, 0.6]), "rot": rot}
        else:
            kind = "mlstm"
            mixer = {"heads": pick([1, 2, 3, 5]), "dim": pick([4, 8, 16, 18, 40, 64, 104, 128, 200, 320]),
                     "vdim": pick([7, 8, 17, 32, 64, 136, 264]), "gate_cap": float(pick([1.0, 5.0, 15.0]))}
        draw = rng.random()
        mlp = None
        if draw < 0.45:
            experts = pick([1, 3, 4, 8, 20])
            mlp = {"kind": "moe", "expert": {"ff": pick([8, 20, 64, 128])},
                   "router": {"experts": experts, "top": int(rng.integers(1, min(experts, 5) + 1))}}
            if rng.random() < 0.6:
                mlp["shared"] = {"ff": pick([8, 36, 96])}
        elif draw < 0.85:
            mlp = {"kind": "dense", "ff": pick([8, 20, 100, 128]), "limit": float(pick([0.3, 1.0, 7.0]))}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    config = {"architecture": "Manatar", "vocab": pick([97, 256, 300]), "width": width,
              "norm": {"eps": float(pick([1e-6, 1e-5, 1e-3]))}, "layers": layers,
              "residual_mult": float(pick([0.3, 0.7, 1.0, -0.5]))}
    if rng.random() < 0.7:
        config["embedding"] = {"bigram": {"buckets": pick([1, 7, 100, 997]), "mul_prev": pick([1, 29, -9]),
                                          "mul_cur": pick([19, 1, 1000003])}}
    return config


@pytest.mark.parametrize("seed", range(int(os.environ.get("HELIX_SWEEP_SEEDS", "12"))))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configuration_in_mixed_batches(seed, dtype, model_root):
    config = draw_config(seed)
    folder = os.path.join(model_root, f"manatar_sweep_{seed}_{dtype}")
    storage = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    write_model_folder(folder, config, tensors_for(config, 90 + seed, storage))
    # every third model also gets a long request fed in long portions
    long_one = seed % 3 == 0
    lengths = (1, 7, 45, 130, 77) + ((400,) if long_one else ())
    requests = {f"r{index}": random_tokens(config["vocab"], length, seed=seed * 10 + index)
                for index, length in enumerate(lengths)}
    expected = Expected(folder, PlainManatar(folder, dtype), dtype, requests)
    steps = traces.mixed(requests, max_live=3, seed=seed,
                         chunk_choices=(2, 3, 7, 16, 33, 64) + ((300, 129) if long_one else ()))
    page = int(np.random.default_rng(seed).choice([8, 16]))
    pages = -(-traces.live_token_need(steps, round_to=page) // page)
    harness = Harness(folder, dtype, page, num_pages=pages, max_requests=3, max_tokens=1024)
    positions = {}
    for step in steps:
        rows = traces.labels(step, positions)
        out = harness.run([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        for name in step["end"]:
            harness.end(name)
        check_rows(out, expected, rows, f"seed {seed} step {step['step']}")
    harness.cache.check()
    assert not harness.cache.live_requests()

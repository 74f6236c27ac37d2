"""Randomly drawn Pizilix configurations through the engine against the plain implementation: the
order and number of layers, loops over any stretch of them, every size of the two mixers (heads,
grouped key/value heads, head sizes up to 288, chunks of 1 to 300 positions or none, rotation of
some or all coordinates with and without stretched frequencies, levels from far below to far above
the scores; widths of 8 to 272 channels in 1 to 16 blocks, filters of 1 to 6 taps), layers without a
feed-forward, with and without a level for the logits, and every model is replayed as mixed
batches over a pool made for its live requests only."""
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
from pizilix_configs import tensors_for
from plain_pizilix import PlainPizilix
from test_pizilix_model_gpu import Expected, check_rows

pytestmark = pytest.mark.gpu


def draw_config(seed: int):
    rng = np.random.default_rng(8000 + seed)
    pick = lambda values: values[int(rng.integers(0, len(values)))]
    width = pick([40, 64, 72, 100, 128, 136, 256])
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        if rng.random() < 0.5:
            dim, kv_heads = pick([4, 8, 20, 32, 64, 80, 128, 288]), pick([1, 1, 2, 3])
            rot = {"base": float(pick([100.0, 10000.0, 500000.0])),
                   "dims": pick([d for d in (2, dim // 2, dim) if d % 2 == 0 and d > 0])}
            if rng.random() < 0.6:
                rot["scaling"] = {"factor": float(pick([1.5, 4.0, 40.0])),
                                  "original": pick([8, 32, 64, 512]),
                                  "fast": float(pick([1.0, 4.0, 32.0])),
                                  "slow": float(pick([0.25, 1.0, 2.0]))}
            mixer = {"heads": kv_heads * pick([1, 2, 3, 4, 8]), "kv_heads": kv_heads, "dim": dim,
                     "vdim": dim, "scale": pick([1.0, 2.0, 4.0]) / math.sqrt(dim), "rot": rot}
            if rng.random() < 0.85:
                mixer["mask"] = {"size": pick([1, 2, 5, 16, 17, 31, 40, 64, 90, 128, 300])}
            if rng.random() < 0.7:
                mixer["softcap"] = float(pick([0.5, 2.0, 8.0, 30.0, 1000.0]))
            kind = "attention"
        else:
            blocks = pick([1, 2, 3, 4, 16])
            mixer = {"width": blocks * pick([8, 10, 16, 17, 40, 64, 136]) if blocks < 16 else
                     16 * pick([1, 8, 17]), "blocks": blocks, "conv": pick([1, 2, 3, 4, 6])}
            kind = "rglru"
        mlp = None if rng.random() < 0.2 else {"kind": "dense", "ff": pick([8, 20, 48, 100, 128, 256])}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    config = {"architecture": "Pizilix", "vocab": pick([97, 256, 300]), "width": width,
              "norm": {"eps": float(pick([1e-6, 1e-5, 1e-3]))}, "layers": layers}
    if rng.random() < 0.7:
        config["logit_softcap"] = float(pick([1.0, 5.0, 30.0]))
    if rng.random() < 0.6:
        start = int(rng.integers(0, len(layers)))
        config["loop"] = {"start": start, "stop": int(rng.integers(start + 1, len(layers) + 1)),
                          "times": pick([1, 2, 3])}
    return config


@pytest.mark.parametrize("seed", range(int(os.environ.get("HELIX_SWEEP_SEEDS", "12"))))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configuration_in_mixed_batches(seed, dtype, model_root):
    config = draw_config(seed)
    folder = os.path.join(model_root, f"pizilix_sweep_{seed}_{dtype}")
    storage = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    write_model_folder(folder, config, tensors_for(config, 90 + seed, storage))
    # every third model also gets a long request fed in long portions
    long_one = seed % 3 == 0
    lengths = (1, 7, 45, 130, 77) + ((400,) if long_one else ())
    requests = {f"r{index}": random_tokens(config["vocab"], length, seed=seed * 10 + index)
                for index, length in enumerate(lengths)}
    expected = Expected(folder, PlainPizilix(folder, dtype), dtype, requests)
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

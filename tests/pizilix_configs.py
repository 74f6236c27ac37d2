"""Small Pizilix configurations for the tests and how their model folders are made.

They differ in every size and constant, and inside a model the layers differ too:

* ``mixed``: both mixers, a loop of three passes over two attention layers (one without a
  feed-forward), chunks of 21 and 33 positions over pages of 8, stretched rotary frequencies whose
  original length (24) the prompts pass, scores and logits that run into a level, a filter of four
  taps over five blocks of channels and one of a single tap over one block.
* ``plain``: no loop, no levels, no stretched frequencies, one attention layer without chunks,
  as many key/value heads as query heads, chunks (5) smaller than a page.
* ``fast``: shapes the tensor-core kernels take (width 256, heads of 64 and 128, blocks of 128),
  sharp attention in chunks of 96 and 200, prompts of hundreds of tokens.
* ``odd``: sizes no fast kernel takes: width 72, an odd vocabulary, heads of 10 of which 4
  coordinates turn, three query heads on one key/value head, blocks of 15 channels, a level the
  scores run far into.

Weights are drawn so that nothing is trivial: attention is sharp, biases are not zero, channels
forget within a token or keep their state for a thousand.
"""
from __future__ import annotations

import math
import os

import numpy as np
import torch

from helix_runtime_b200.weights.random_init import write_model_folder


def _attention(heads, kv_heads, dim, chunk, rot_dims, base, scaling=None, softcap=None, ff=None,
               sharp=2.0):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
             "scale": sharp / math.sqrt(dim), "rot": rot}
    if softcap is not None:
        mixer["softcap"] = softcap
    if chunk is not None:
        mixer["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": mixer,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _rglru(width, blocks, conv, ff=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


CONFIGS = {
    "mixed": {
        "architecture": "Pizilix", "vocab": 211, "width": 96, "norm": {"eps": 1e-5},
        "logit_softcap": 6.0, "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [_rglru(120, 5, 4, 80),
                   _attention(4, 2, 24, 21, 12, 10000.0, (4.0, 24, 8.0, 1.0), 9.0, 80),
                   _attention(3, 1, 16, 33, 16, 500.0),
                   _rglru(64, 1, 1, 48)],
    },
    "plain": {
        "architecture": "Pizilix", "vocab": 300, "width": 128, "norm": {"eps": 1e-6},
        "layers": [_attention(4, 4, 32, None, 32, 10000.0, ff=96),
                   _rglru(64, 8, 2),
                   _attention(2, 2, 16, 5, 8, 300.0, ff=48)],
    },
    "fast": {
        "architecture": "Pizilix", "vocab": 640, "width": 256, "norm": {"eps": 1e-5},
        "logit_softcap": 20.0, "loop": {"start": 0, "stop": 2, "times": 2},
        "layers": [_rglru(256, 2, 4, 256),
                   _attention(8, 2, 64, 96, 32, 20000.0, (6.0, 128, 16.0, 2.0), 12.0, 384, sharp=4.0),
                   _attention(4, 1, 128, 200, 128, 10000.0, None, 30.0, 256, sharp=4.0)],
    },
    "odd": {
        "architecture": "Pizilix", "vocab": 101, "width": 72, "norm": {"eps": 1e-4},
        "logit_softcap": 3.0, "loop": {"start": 1, "stop": 3, "times": 2},
        "layers": [_rglru(90, 6, 3, 30),
                   _attention(3, 1, 10, 7, 4, 77.0, (3.0, 10, 2.0, 0.25), 1.5, 20),
                   _rglru(36, 2, 5)],
    },
}
PAGE_SIZE = {"mixed": 8, "plain": 16, "fast": 16, "odd": 8}
SEED = {"mixed": 71, "plain": 72, "fast": 73, "odd": 74}


def tensors_for(config: dict, seed: int, storage_dtype: torch.dtype):
    rng = np.random.default_rng(seed)
    width = config["width"]

    def store(values):
        return torch.tensor(np.asarray(values), dtype=torch.float32).to(storage_dtype)

    def matrix(rows, columns, gain=1.0):
        return store(rng.normal(size=(rows, columns)) * gain / math.sqrt(columns))

    def vector(shape, spread, mean=0.0):
        return store(mean + spread * rng.normal(size=shape))

    # the table is the head as well: its rows are of the length that gives logits of spread one
    # or two behind the final norm
    tensors = {"embed": matrix(config["vocab"], width, 1.5), "final.norm": vector(width, 0.2)}
    for index, layer in enumerate(config["layers"]):
        prefix, mixer = f"l{index}", layer["mixer"]
        for name in ("norm1",) + (("norm2",) if layer["mlp"] else ()):
            tensors[f"{prefix}.{name}"] = vector(width, 0.2)
        if layer["type"] == "attention":
            heads, kv_heads, dim = (mixer[k] for k in ("heads", "kv_heads", "dim"))
            tensors[f"{prefix}.mix.q"] = matrix(heads * dim, width, 1.2)
            tensors[f"{prefix}.mix.k"] = matrix(kv_heads * dim, width, 1.2)
            tensors[f"{prefix}.mix.o"] = matrix(width, heads * dim, 0.7)
        else:
            w, blocks, taps = mixer["width"], mixer["blocks"], mixer["conv"]
            size = w // blocks
            for name in ("y", "x"):
                tensors[f"{prefix}.mix.{name}"] = matrix(w, width, 1.2)
                tensors[f"{prefix}.mix.{name}.b"] = vector(w, 0.3)
            tensors[f"{prefix}.mix.conv"] = store(rng.normal(size=(w, taps)) / math.sqrt(taps))
            tensors[f"{prefix}.mix.conv.b"] = vector(w, 0.3)
            for name in ("ra", "ri"):
                tensors[f"{prefix}.mix.{name}"] = store(rng.normal(size=(blocks, size, size))
                                                        * 1.5 / math.sqrt(size))
                tensors[f"{prefix}.mix.{name}.b"] = vector((blocks, size), 0.5)
            tensors[f"{prefix}.mix.lam"] = store(rng.uniform(-8.0, 1.0, size=w))
            tensors[f"{prefix}.mix.o"] = matrix(width, w, 1.5)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            tensors[f"{prefix}.mlp.gate"] = matrix(ff, width, 1.5)
            tensors[f"{prefix}.mlp.up"] = matrix(ff, width, 1.5)
            tensors[f"{prefix}.mlp.down"] = matrix(width, ff, 0.7)
    return tensors


def make_folder(directory: str, name: str, storage_dtype: str = "float32") -> str:
    path = os.path.join(directory, f"pizilix_{name}_{storage_dtype}")
    if not os.path.exists(os.path.join(path, "model.safetensors")):
        dtype = torch.bfloat16 if storage_dtype == "bfloat16" else torch.float32
        write_model_folder(path, CONFIGS[name], tensors_for(CONFIGS[name], SEED[name], dtype))
    return path

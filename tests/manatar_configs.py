"""Small Manatar configurations for the tests and how their model folders are made.

They differ in every size and constant, and inside a model the layers differ too:

* ``mixed``: both mixers in turn, two layers that use an earlier layer's keys and values (one
  right behind it, one three layers on, each with a filter, scale and balance of its own), a
  layer without a feed-forward, a filter of one tap, stretched frequencies whose original length
  (24) the prompts pass, a dense and three routed feed-forwards with and without a shared expert,
  a table of pairs with a negative factor.
* ``plain``: no table of pairs, no stretched frequencies, as many key/value heads as query heads,
  values narrower than both maps together, a router that uses one expert, residual factor 1.
* ``fast``: shapes the tensor-core kernels take (width 256, maps of 64 and 32, values of 128 and 64,
  matrices of 64 by 128 and 136 by 48), prompts of hundreds of tokens.
* ``odd``: sizes no fast kernel takes: width 72, an odd vocabulary, maps of 9 and 10 of which 4
  coordinates turn, values of 14 and 7, three query heads on one key/value head, filters of five
  taps, matrices of 18 by 7, every expert chosen, a table of pairs with one bucket, a negative
  residual factor and a balance below zero.

Weights are drawn so that nothing is trivial: attention is sharp, biases are not zero, heads of the
recurrence forget within a token or keep their state for a thousand, and the routers' biases are
far enough apart that few choices are close.
"""
from __future__ import annotations

import math
import os

import numpy as np
import torch

from helix_runtime_b200.weights.random_init import write_model_folder


def _attention(heads, kv_heads, dim, vdim, conv, diff, rot_dims, base, scaling=None, kv_from=None,
               mlp=None, sharp=2.0):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
             "diff": diff, "scale": sharp / math.sqrt(dim), "rot": rot}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _mlstm(heads, dim, vdim, gate_cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap},
            "mlp": mlp}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


CONFIGS = {
    "mixed": {
        "architecture": "Manatar", "vocab": 211, "width": 96, "norm": {"eps": 1e-5},
        "residual_mult": 0.6, "embedding": {"bigram": {"buckets": 37, "mul_prev": 13, "mul_cur": -5}},
        "layers": [_attention(4, 2, 24, 40, 4, 0.25, 16, 10000.0, (4.0, 24, 8.0, 1.0), mlp=_dense(80, 0.7)),
                   _attention(4, 2, 24, 40, 2, 0.6, 16, 10000.0, (4.0, 24, 8.0, 1.0), kv_from=0, sharp=3.0),
                   _mlstm(3, 16, 24, 6.0, _moe(6, 2, 40, 56)),
                   _attention(4, 2, 24, 40, 3, 0.1, 16, 10000.0, (4.0, 24, 8.0, 1.0), kv_from=0,
                              mlp=_moe(5, 3, 48)),
                   _attention(2, 1, 20, 20, 1, 0.4, 20, 500.0, mlp=_moe(4, 1, 32, 24))],
    },
    "plain": {
        "architecture": "Manatar", "vocab": 300, "width": 128, "norm": {"eps": 1e-6},
        "residual_mult": 1.0,
        "layers": [_attention(4, 4, 32, 32, 3, 0.35, 32, 10000.0, mlp=_moe(7, 1, 64, 96)),
                   _mlstm(2, 32, 32, 15.0, _dense(96, 2.0)),
                   _mlstm(4, 8, 16, 3.0)],
    },
    "fast": {
        "architecture": "Manatar", "vocab": 640, "width": 256, "norm": {"eps": 1e-5},
        "residual_mult": 0.5, "embedding": {"bigram": {"buckets": 500, "mul_prev": 29, "mul_cur": 7}},
        "layers": [_attention(4, 2, 64, 128, 4, 0.3, 64, 20000.0, (6.0, 128, 16.0, 2.0),
                              mlp=_dense(384, 1.5), sharp=1.5),
                   _mlstm(2, 64, 128, 12.0, _moe(8, 2, 128, 128)),
                   _attention(4, 2, 64, 128, 4, 0.2, 64, 20000.0, (6.0, 128, 16.0, 2.0), kv_from=0,
                              mlp=_moe(8, 3, 128), sharp=1.5),
                   _mlstm(3, 136, 48, 15.0, _dense(256, 0.5)),
                   _attention(8, 1, 32, 64, 2, 0.5, 24, 10000.0, mlp=_moe(6, 4, 64, 64))],
    },
    "odd": {
        "architecture": "Manatar", "vocab": 101, "width": 72, "norm": {"eps": 1e-4},
        "residual_mult": -0.8, "embedding": {"bigram": {"buckets": 1, "mul_prev": 2, "mul_cur": 3}},
        "layers": [_attention(3, 1, 10, 14, 5, 0.2, 4, 77.0, (3.0, 10, 2.0, 0.25), mlp=_moe(5, 5, 20, 12)),
                   _mlstm(3, 18, 7, 4.0, _dense(30, 0.4)),
                   _attention(2, 2, 9, 7, 3, -0.3, 4, 300.0, mlp=_dense(20, 1.0)),
                   _attention(2, 2, 9, 7, 5, 0.8, 4, 300.0, kv_from=2)],
    },
}
PAGE_SIZE = {"mixed": 8, "plain": 16, "fast": 16, "odd": 8}
# Distance of neighbouring router biases: what decides how many tokens are close calls.  The model with
# the longest requests has the widest.
SPACING = {"mixed": 1.4, "plain": 1.2, "fast": 2.0, "odd": 1.2}
SEED = {"mixed": 81, "plain": 82, "fast": 83, "odd": 84}


def tensors_for(config: dict, seed: int, storage_dtype: torch.dtype, spacing: float = 1.2):
    rng = np.random.default_rng(seed)
    width = config["width"]

    def store(values):
        return torch.tensor(np.asarray(values), dtype=torch.float32).to(storage_dtype)

    def matrix(rows, columns, gain=1.0):
        return store(rng.normal(size=(rows, columns)) * gain / math.sqrt(columns))

    def vector(shape, spread, mean=0.0):
        return store(mean + spread * rng.normal(size=shape))

    tensors = {"embed": store(rng.normal(size=(config["vocab"], width))),
               "head": matrix(config["vocab"], width, 1.5), "final.norm": vector(width, 0.2, 1.0)}
    pairs = (config.get("embedding") or {}).get("bigram")
    if pairs:
        tensors["bigram"] = store(0.7 * rng.normal(size=(pairs["buckets"] + 1, width)))

    def small_feed_forward(prefix, ff):
        tensors[f"{prefix}.gate"] = matrix(ff, width, 1.5)
        tensors[f"{prefix}.up"] = matrix(ff, width, 1.5)
        tensors[f"{prefix}.down"] = matrix(width, ff)

    for index, layer in enumerate(config["layers"]):
        prefix, mixer, mlp = f"l{index}", layer["mixer"], layer["mlp"]
        for name in ("norm1",) + (("norm2",) if mlp else ()):
            tensors[f"{prefix}.{name}"] = vector(width, 0.2, 1.0)
        mix = f"{prefix}.mix"
        if layer["type"] == "attention":
            heads, groups, dim, vdim, taps = (mixer[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
            sources = [("q", heads * 2 * dim)]
            if mixer.get("kv_from") is None:
                sources += [("k", groups * 2 * dim), ("v", groups * vdim)]
            for name, rows in sources:
                tensors[f"{mix}.{name}"] = matrix(rows, width, 1.2)
                tensors[f"{mix}.{name}.b"] = vector(rows, 0.3)
                tensors[f"{mix}.{name}.conv"] = store(rng.normal(size=(rows, taps)) / math.sqrt(taps))
                if name != "v":
                    tensors[f"{mix}.{name}.norm"] = vector(dim, 0.2, 1.0)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                tensors[f"{mix}.{name}"] = vector(dim, 0.8 / math.sqrt(dim))
            tensors[f"{mix}.g"] = matrix(heads * vdim, width, 1.5)
            tensors[f"{mix}.o"] = matrix(width, heads * vdim)
            tensors[f"{mix}.o.b"] = vector(width, 0.2)
        else:
            heads, dim, vdim = (mixer[k] for k in ("heads", "dim", "vdim"))
            for name, rows in (("q", heads * dim), ("k", heads * dim), ("v", heads * vdim),
                               ("g", heads * vdim), ("i", heads), ("f", heads)):
                tensors[f"{mix}.{name}"] = matrix(rows, width, 1.2)
            tensors[f"{mix}.i.b"] = vector(heads, 1.0)
            tensors[f"{mix}.f.b"] = store(np.resize([7.0, 1.0, 4.0, -2.0], heads) + 0.1 * rng.normal(size=heads))
            tensors[f"{mix}.norm"] = vector(heads * vdim, 0.2, 1.0)
            tensors[f"{mix}.o"] = matrix(width, heads * vdim)
        if mlp and mlp["kind"] == "dense":
            small_feed_forward(f"{prefix}.mlp", mlp["ff"])
        elif mlp:
            experts = mlp["router"]["experts"]
            tensors[f"{prefix}.mlp.router"] = matrix(experts, width, 0.25)
            tensors[f"{prefix}.mlp.router.b"] = store(rng.permutation(experts) * spacing)
            for expert in range(experts):
                small_feed_forward(f"{prefix}.mlp.e{expert}", mlp["expert"]["ff"])
            if mlp.get("shared"):
                small_feed_forward(f"{prefix}.mlp.shared", mlp["shared"]["ff"])
    return tensors


def make_folder(directory: str, name: str, storage_dtype: str = "float32") -> str:
    path = os.path.join(directory, f"manatar_{name}_{storage_dtype}")
    if not os.path.exists(os.path.join(path, "model.safetensors")):
        dtype = torch.bfloat16 if storage_dtype == "bfloat16" else torch.float32
        write_model_folder(path, CONFIGS[name],
                           tensors_for(CONFIGS[name], SEED[name], dtype, SPACING[name]))
    return path

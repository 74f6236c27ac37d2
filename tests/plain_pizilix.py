"""Plain, slow implementation of the Pizilix decoder: whole sequences, no cache, NumPy in
double precision, one function per mechanism.  It shares no code with the engine (own
safetensors reader, own order of layers, own masks, own recurrence written token by token).

Notation.  One residual row per token, ``x <- x + f(norm(x))`` for the mixer and then for the
feed-forward, ``norm(x) = x / sqrt(mean(x^2) + eps) * (1 + w)``; the residual starts as the
token's row of the table.  A stretch of layers may run several times; before every repeat the
start value is added to the residual once more.

Mixers (``h`` is the normed input ``[T, W]``):

* attention: ``q = Wq h`` in heads, ``k = Wk h`` in key/value heads, the VALUES are ``k`` as
  projected; q and k turn by their position over their first ``dims`` coordinates (pairs ``2m,
  2m + 1``), with frequencies stretched for contexts beyond a trained length; the score is
  ``cap * tanh(scale * (q . k) / cap)``; position ``i`` sees ``j <= i`` of its own chunk of
  ``size`` positions; the weights are ``exp(s) / (1 + sum exp(s))``.
* rglru: ``y = gelu_tanh(Wy h + by)``, ``u`` a causal per-channel filter with bias over ``Wx h +
  bx``; per block of channels ``r = sigmoid(Ra u + ba)``, ``i = sigmoid(Ri u + bi)``; per channel
  ``log a = -8 r softplus(lam)``, ``S_t = a S_(t-1) + sqrt(1 - a^2) i u``; ``Wo (S * y)``.

Feed-forward: ``Wdown (silu(Wgate h) * (Wup h))``.  Output: the norm, the table as the head, and
``cap * tanh(logits / cap)``.

``precision="bfloat16"`` rounds activations to bfloat16 where a bfloat16 engine stores them
(norm outputs, projections before their biases, rotated heads, filtered rows, attention output, the recurrence's
gated output, the feed-forward's activation); sums, scores, recurrences and the residual stay
in double.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Callable, Dict, List, Optional, Tuple

import numpy as np


def read_safetensors(path: str) -> Dict[str, np.ndarray]:
    with open(path, "rb") as source:
        (length,) = struct.unpack("<Q", source.read(8))
        header = json.loads(source.read(length).decode("utf-8"))
        payload = source.read()
    header.pop("__metadata__", None)
    tensors = {}
    for name, record in header.items():
        begin, end = record["data_offsets"]
        raw = payload[begin:end]
        if record["dtype"] == "F32":
            value = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif record["dtype"] == "BF16":
            bits = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << np.uint32(16)
            value = bits.view(np.float32).astype(np.float64)
        else:
            raise ValueError(f"unsupported dtype {record['dtype']}")
        tensors[name] = value.reshape(tuple(record["shape"]))
    return tensors


def to_bfloat16(values: np.ndarray) -> np.ndarray:
    """Round to the nearest bfloat16 (ties to even), returned as float64."""
    bits = np.asarray(values, dtype=np.float32).view(np.uint32).astype(np.uint64)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16
    return rounded.astype(np.uint32).view(np.float32).astype(np.float64).reshape(np.shape(values))


def identity(values: np.ndarray) -> np.ndarray:
    return values


# ------------------------------------------------------------------- small functions

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm_one_plus(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * (1.0 + weight)


def softcap(z: np.ndarray, cap: Optional[float]) -> np.ndarray:
    return z if cap is None else cap * np.tanh(z / cap)


# ------------------------------------------------------------------- mechanisms

def rotary_frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[np.ndarray, float]:
    """The ``dims / 2`` frequencies and the factor on sine and cosine."""
    frequencies, amplitude = [], 1.0
    for m in range(dims // 2):
        f = base ** (-2.0 * m / dims)
        if scaling is not None:
            def place(turns):
                return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) \
                    / (2.0 * math.log(base))
            lo = max(math.floor(place(scaling["fast"])), 0)
            hi = min(math.ceil(place(scaling["slow"])), dims - 1)
            ramp = min(max((m - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * ramp + f * (1.0 - ramp)
        frequencies.append(f)
    if scaling is not None:
        amplitude = 0.1 * math.log(scaling["factor"]) + 1.0
    return np.array(frequencies), amplitude


def rotate_neighbours(x: np.ndarray, positions: np.ndarray, frequencies: np.ndarray,
                      amplitude: float) -> np.ndarray:
    """``x [T, heads, D]``: coordinates ``2m`` and ``2m + 1`` turn by ``position * f[m]``; what
    lies behind the last pair passes."""
    out = x.copy()
    for m, f in enumerate(frequencies):
        cos = (np.cos(positions * f) * amplitude)[:, None]
        sin = (np.sin(positions * f) * amplitude)[:, None]
        u, v = x[:, :, 2 * m], x[:, :, 2 * m + 1]
        out[:, :, 2 * m] = u * cos - v * sin
        out[:, :, 2 * m + 1] = v * cos + u * sin
    return out


def chunked_attention(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float,
                      cap: Optional[float], size: Optional[int], sink: bool = True) -> np.ndarray:
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]``: position ``i`` sees ``j <= i`` with
    ``i // size == j // size`` (``size`` None: every ``j <= i``); the softmax's denominator holds
    one more term ``exp(0)``."""
    length, heads, _ = q.shape
    per_group = heads // k.shape[1]
    out = np.zeros((length, heads, v.shape[2]))
    for head in range(heads):
        group = head // per_group
        for i in range(length):
            seen = [j for j in range(i + 1) if size is None or j // size == i // size]
            scores = softcap((k[seen, group] @ q[i, head]) * scale, cap)
            top = max(scores.max(), 0.0)
            weights = np.exp(scores - top)
            total = weights.sum() + (math.exp(-top) if sink else 0.0)
            out[i, head] = (weights / total) @ v[seen, group]
    return out


def causal_filter_bias(u: np.ndarray, taps: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """``u [T, C]``, ``taps [C, n]`` with the last column on the token itself, zeros before the
    sequence: ``y[t, c] = bias[c] + sum_j taps[c, j] u[t - (n - 1) + j, c]``."""
    length, n = u.shape[0], taps.shape[1]
    out = np.tile(bias[None, :], (length, 1)).astype(np.float64)
    for t in range(length):
        for j in range(n):
            source = t - (n - 1) + j
            if source >= 0:
                out[t] += taps[:, j] * u[source]
    return out


def block_products(u: np.ndarray, matrices: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """``u [T, C]`` in as many equal parts as there are square matrices ``[B, n, n]``; part ``b``
    is multiplied by its own matrix, ``bias [B, n]`` is added."""
    parts = np.split(u, matrices.shape[0], axis=1)
    return np.concatenate([part @ matrix.T + add
                           for part, matrix, add in zip(parts, matrices, bias)], axis=1)


def gated_linear_recurrence(u: np.ndarray, r: np.ndarray, i: np.ndarray, lam: np.ndarray) -> np.ndarray:
    """``S_t = a S_(t-1) + sqrt(1 - a^2) i u`` with ``log a = -8 r softplus(lam)``, every channel
    by itself, token by token from zero."""
    out, state = np.zeros_like(u), np.zeros(u.shape[1])
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        state = np.exp(log_a) * state + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = state
    return out


# ------------------------------------------------------------------------ the model

class PlainPizilix:
    def __init__(self, folder: str, precision: str = "float32") -> None:
        with open(os.path.join(folder, "config.json")) as source:
            self.config = json.load(source)
        self.w = read_safetensors(os.path.join(folder, "model.safetensors"))
        self.round: Callable[[np.ndarray], np.ndarray] = \
            to_bfloat16 if precision == "bfloat16" else identity
        self.eps = float(self.config["norm"]["eps"])
        self.after_layer: Optional[Callable[[int, np.ndarray], None]] = None

    def linear(self, name: str, x: np.ndarray) -> np.ndarray:
        return x @ self.w[name].T

    def attention_mixer(self, prefix: str, sizes: dict, h: np.ndarray, positions: np.ndarray) -> np.ndarray:
        heads, groups, dim, length = sizes["heads"], sizes["kv_heads"], sizes["dim"], h.shape[0]
        q = self.round(self.linear(f"{prefix}.q", h)).reshape(length, heads, dim)
        k = self.round(self.linear(f"{prefix}.k", h)).reshape(length, groups, dim)
        v = k
        rot = sizes["rot"]
        turns = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q = self.round(rotate_neighbours(q, positions, *turns))
        k = self.round(rotate_neighbours(k, positions, *turns))
        mask = sizes.get("mask") or {}
        out = chunked_attention(q, k, v, sizes["scale"], sizes.get("softcap"), mask.get("size"))
        return self.linear(f"{prefix}.o", self.round(out.reshape(length, heads * dim)))

    def recurrent_mixer(self, prefix: str, sizes: dict, h: np.ndarray) -> np.ndarray:
        y = gelu_tanh(self.round(self.linear(f"{prefix}.y", h)) + self.w[f"{prefix}.y.b"])
        x = self.round(self.linear(f"{prefix}.x", h)) + self.w[f"{prefix}.x.b"]
        u = self.round(causal_filter_bias(x, self.w[f"{prefix}.conv"], self.w[f"{prefix}.conv.b"]))
        r = sigmoid(block_products(u, self.w[f"{prefix}.ra"], self.w[f"{prefix}.ra.b"]))
        i = sigmoid(block_products(u, self.w[f"{prefix}.ri"], self.w[f"{prefix}.ri.b"]))
        state = gated_linear_recurrence(u, r, i, self.w[f"{prefix}.lam"])
        return self.linear(f"{prefix}.o", self.round(state * y))

    def mixer(self, index: int, layer: dict, h: np.ndarray, positions: np.ndarray) -> np.ndarray:
        prefix, sizes = f"l{index}.mix", layer["mixer"]
        if layer["type"] == "attention":
            return self.attention_mixer(prefix, sizes, h, positions)
        if layer["type"] == "rglru":
            return self.recurrent_mixer(prefix, sizes, h)
        raise ValueError(f"unknown layer type {layer['type']!r}")

    def feed_forward(self, index: int, h: np.ndarray) -> np.ndarray:
        prefix = f"l{index}.mlp"
        hidden = silu(self.linear(f"{prefix}.gate", h)) * self.linear(f"{prefix}.up", h)
        return self.linear(f"{prefix}.down", self.round(hidden))

    def layer_order(self) -> List[Tuple[int, bool]]:
        """``(layer, add the start value first)`` in the order the layers run."""
        count, loop = len(self.config["layers"]), self.config.get("loop")
        if not loop:
            return [(layer, False) for layer in range(count)]
        order = [(layer, False) for layer in range(loop["start"])]
        for turn in range(loop["times"]):
            order += [(layer, turn > 0 and layer == loop["start"])
                      for layer in range(loop["start"], loop["stop"])]
        return order + [(layer, False) for layer in range(loop["stop"], count)]

    def logits(self, tokens) -> np.ndarray:
        return self.forward(tokens).astype(np.float32)

    def hidden_states(self, tokens) -> List[np.ndarray]:
        """The residual after every run of a layer."""
        states: List[np.ndarray] = []
        self.after_layer = lambda run, x: states.append(x.copy())
        try:
            self.forward(tokens)
        finally:
            self.after_layer = None
        return states

    def forward(self, tokens) -> np.ndarray:
        """Logits ``[T, vocab]`` of one whole sequence from position 0."""
        tokens = np.asarray(tokens, dtype=np.int64)
        positions = np.arange(len(tokens), dtype=np.float64)
        start = self.w["embed"][tokens]
        x = start.copy()
        for run, (index, again) in enumerate(self.layer_order()):
            layer, prefix = self.config["layers"][index], f"l{index}"
            if again:
                x = x + start
            h = self.round(rms_norm_one_plus(x, self.w[f"{prefix}.norm1"], self.eps))
            x = x + self.mixer(index, layer, h, positions)
            if layer.get("mlp") is not None:
                h = self.round(rms_norm_one_plus(x, self.w[f"{prefix}.norm2"], self.eps))
                x = x + self.feed_forward(index, h)
            if self.after_layer is not None:
                self.after_layer(run, x)
        final = self.round(rms_norm_one_plus(x, self.w["final.norm"], self.eps))
        return softcap(final @ self.w["embed"].T, self.config.get("logit_softcap"))

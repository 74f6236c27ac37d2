"""Plain, slow implementation of the Manatar decoder: whole sequences, no cache, NumPy in double
precision, one function per mechanism.  It shares no code with the engine (own safetensors
reader, own frequencies, own masks, own recurrence written token by token).

Notation.  ``x`` is a token's residual.  It starts as the token's row of the table plus a row of a
second table that the pair (previous token, token) picks.  A layer is ``x <- x + c N1(mixer(x))``,
then, when it has a feed-forward, ``x <- x + c N2(ff(x))``: the norms ``N(y) = y / sqrt(mean(y^2) +
eps) * w`` sit behind the sublayers, which read ``x`` itself.

Mixers:

* attention: two score maps per head over one value.  ``q``, ``k``, ``v`` are projections with
  biases, each channel filtered over time; per head and map q and k pass an RMS norm and turn by
  their position (neighbouring coordinates, frequencies stretched for long contexts); two causal
  softmaxes give ``a1`` and ``a2``; ``o = a1 - lam a2`` over its root mean square times ``1 -
  diff``, with ``lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff``; times ``sigmoid(G x)``; the output
  matrix with its bias.  A layer may use an earlier layer's keys and values.
* mlstm: one matrix ``S`` and one vector ``n`` per head with exponential input gates and
  sigmoid forget gates, kept in the scale ``exp(-m)`` of a running maximum.

Feed-forwards: a clamped gated layer, or experts behind a router that is a softmax over the
chosen logits, with an expert that every token uses.

``precision="bfloat16"`` rounds activations to bfloat16 where a bfloat16 engine stores them
(sublayer inputs, projections before their biases, rotated heads, filtered values, attention
output of each map, the gated heads, what lies between a feed-forward's products); sums, scores,
gates of the recurrence, recurrences and the residual stay in double.
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
    return np.exp(-np.logaddexp(0.0, -np.asarray(z, dtype=np.float64)))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return unit_rms(x, eps) * weight


def pair_rows(tokens: np.ndarray, buckets: int, mul_prev: int, mul_cur: int) -> np.ndarray:
    """Row of the second table for every token: the pair's bucket, the first token's own row."""
    rows = np.empty(len(tokens), dtype=np.int64)
    rows[0] = buckets
    for t in range(1, len(tokens)):
        rows[t] = (int(tokens[t - 1]) * mul_prev + int(tokens[t]) * mul_cur) % buckets
    return rows


def causal_filter(u: np.ndarray, taps: np.ndarray) -> np.ndarray:
    """``y[t, c] = sum_j taps[c, j] u[t - J + 1 + j, c]`` with zeros in front of the sequence."""
    length, count = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((count - 1, u.shape[1])), u], axis=0)
    out = np.zeros_like(u)
    for j in range(count):
        out += padded[j:j + length] * taps[:, j]
    return out


def rotary_frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[np.ndarray, float]:
    """Frequencies of the ``dims / 2`` pairs and the factor on sine and cosine."""
    plain = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return plain, 1.0

    def pair_of(turns: float) -> float:
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    low = max(math.floor(pair_of(scaling["fast"])), 0)
    high = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    blend = np.clip((np.arange(dims // 2) - low) / max(high - low, 0.001), 0.0, 1.0)
    factor = scaling["factor"]
    return plain / factor * blend + plain * (1.0 - blend), 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x: np.ndarray, positions: np.ndarray, frequencies: np.ndarray,
                      amplitude: float) -> np.ndarray:
    """Turn coordinates ``(2i, 2i + 1)`` of ``x [T, ..., D]`` by ``position * frequency_i``."""
    out = x.copy()
    angle = positions[:, None] * frequencies[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (len(frequencies),)
    cosine = (np.cos(angle) * amplitude).reshape(shape)
    sine = (np.sin(angle) * amplitude).reshape(shape)
    turned = 2 * len(frequencies)
    first, second = x[..., 0:turned:2], x[..., 1:turned:2]
    out[..., 0:turned:2] = first * cosine - second * sine
    out[..., 1:turned:2] = second * cosine + first * sine
    return out


def causal_softmax_map(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float) -> np.ndarray:
    """One map of one head: ``q [T, D]``, ``k [T, D]``, ``v [T, E]``."""
    scores = (q @ k.T) * scale
    length = q.shape[0]
    scores[np.triu_indices(length, 1)] = -np.inf
    weights = np.exp(scores - scores.max(axis=1, keepdims=True))
    return (weights / weights.sum(axis=1, keepdims=True)) @ v


def map_balance(lq1, lk1, lq2, lk2, diff: float) -> float:
    """How much of the second map is taken off the first."""
    return float(np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff)


def difference_of_maps(a1: np.ndarray, a2: np.ndarray, lam: float, diff: float,
                       eps: float) -> np.ndarray:
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def lstm_gates(zi: np.ndarray, zf: np.ndarray, cap: float) -> Tuple[np.ndarray, np.ndarray]:
    """Logarithms of the input and forget gates from their pre-activations (biases included)."""
    return cap * np.tanh(zi / cap), -np.logaddexp(0.0, -cap * np.tanh(zf / cap))


def matrix_lstm(q: np.ndarray, k: np.ndarray, v: np.ndarray, log_in: np.ndarray,
                log_forget: np.ndarray, floor: float = 1e-6) -> np.ndarray:
    """One head, token by token: ``q, k [T, D]``, ``v [T, E]``, gates ``[T]``; ``[T, E]``."""
    S = np.zeros((q.shape[1], v.shape[1]))
    n = np.zeros(q.shape[1])
    m = 0.0
    out = np.empty_like(v)
    for t in range(q.shape[0]):
        before, m = m, max(log_forget[t] + m, log_in[t])
        keep, add = math.exp(log_forget[t] + before - m), math.exp(log_in[t] - m)
        S = keep * S + add * np.outer(k[t], v[t])
        n = keep * n + add * k[t]
        out[t] = (q[t] @ S) / (max(abs(float(n @ q[t])), math.exp(-m)) + floor)
    return out


def clamped_gate(gate: np.ndarray, up: np.ndarray, limit: float) -> np.ndarray:
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose_experts(logits: np.ndarray, top: int) -> Tuple[np.ndarray, np.ndarray]:
    """``(chosen [T, top], weights [T, top])``: the largest logits, a softmax over them alone."""
    chosen = np.argsort(-logits, axis=1, kind="stable")[:, :top]
    picked = np.take_along_axis(logits, chosen, axis=1)
    weights = np.exp(picked - picked.max(axis=1, keepdims=True))
    return chosen, weights / weights.sum(axis=1, keepdims=True)


class PlainManatar:
    def __init__(self, directory: str, precision: str = "float64") -> None:
        with open(os.path.join(directory, "config.json"), encoding="utf-8") as source:
            self.config = json.load(source)
        self.w = read_safetensors(os.path.join(directory, "model.safetensors"))
        self.round: Callable[[np.ndarray], np.ndarray] = \
            to_bfloat16 if precision == "bfloat16" else identity
        if precision == "bfloat16":
            for name, value in self.w.items():
                if value.ndim == 2 and not name.endswith(".conv"):
                    self.w[name] = to_bfloat16(value)
        self.eps = self.config["norm"]["eps"]
        self.after_layer: Optional[Callable[[int, np.ndarray], None]] = None
        # smallest distance between the last chosen logit and the best one left out, per token
        self.margins: Optional[np.ndarray] = None

    def linear(self, name: str, x: np.ndarray) -> np.ndarray:
        return x @ self.w[name].T

    def projected(self, name: str, h: np.ndarray, per_head: int) -> np.ndarray:
        """Projection, bias, filter; ``[T, heads, per_head]``."""
        u = self.round(self.linear(name, h)) + self.w[f"{name}.b"]
        u = causal_filter(u, self.w[f"{name}.conv"])
        return u.reshape(h.shape[0], -1, per_head)

    def attention_mixer(self, index: int, sizes: dict, h: np.ndarray, positions: np.ndarray,
                        kept: dict) -> np.ndarray:
        prefix, length = f"l{index}.mix", h.shape[0]
        heads, groups, dim = sizes["heads"], sizes["kv_heads"], sizes["dim"]
        rot = sizes["rot"]
        turns = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))

        def prepared(name: str, count: int) -> np.ndarray:
            x = self.projected(f"{prefix}.{name}", h, dim)        # [T, count * 2, dim]
            x = rms_norm(x, self.w[f"{prefix}.{name}.norm"], self.eps)
            return self.round(rotate_neighbours(x, positions, *turns)).reshape(length, count, 2, dim)
        q = prepared("q", heads)
        if sizes.get("kv_from") is None:
            kept[index] = (prepared("k", groups),
                           self.round(self.projected(f"{prefix}.v", h, sizes["vdim"])))
            k, v = kept[index]
        else:
            k, v = kept[sizes["kv_from"]]
        lam = map_balance(*(self.w[f"{prefix}.{name}"] for name in ("lq1", "lk1", "lq2", "lk2")),
                          sizes["diff"])
        out = np.empty((length, heads, sizes["vdim"]))
        for head in range(heads):
            group = head // (heads // groups)
            a1, a2 = (self.round(causal_softmax_map(q[:, head, part], k[:, group, part], v[:, group],
                                                    sizes["scale"])) for part in (0, 1))
            out[:, head] = difference_of_maps(a1, a2, lam, sizes["diff"], self.eps)
        gate = sigmoid(self.round(self.linear(f"{prefix}.g", h)))
        gated = self.round(out.reshape(length, -1) * gate)
        return self.linear(f"{prefix}.o", gated) + self.w[f"{prefix}.o.b"]

    def lstm_mixer(self, index: int, sizes: dict, h: np.ndarray) -> np.ndarray:
        prefix, length = f"l{index}.mix", h.shape[0]
        heads, dim, vdim = sizes["heads"], sizes["dim"], sizes["vdim"]
        q = self.round(self.linear(f"{prefix}.q", h)).reshape(length, heads, dim) * dim ** -0.5
        k = self.round(self.linear(f"{prefix}.k", h)).reshape(length, heads, dim)
        v = self.round(self.linear(f"{prefix}.v", h)).reshape(length, heads, vdim)
        log_in, log_forget = lstm_gates(self.linear(f"{prefix}.i", h) + self.w[f"{prefix}.i.b"],
                                        self.linear(f"{prefix}.f", h) + self.w[f"{prefix}.f.b"],
                                        sizes["gate_cap"])
        out = np.stack([unit_rms(matrix_lstm(q[:, head], k[:, head], v[:, head], log_in[:, head],
                                             log_forget[:, head]), self.eps)
                        for head in range(heads)], axis=1).reshape(length, heads * vdim)
        gate = sigmoid(self.round(self.linear(f"{prefix}.g", h)))
        return self.linear(f"{prefix}.o", self.round(out * self.w[f"{prefix}.norm"] * gate))

    def small_feed_forward(self, prefix: str, h: np.ndarray) -> np.ndarray:
        hidden = silu(self.linear(f"{prefix}.gate", h)) * self.linear(f"{prefix}.up", h)
        return self.linear(f"{prefix}.down", self.round(hidden))

    def feed_forward(self, index: int, mlp: dict, h: np.ndarray) -> np.ndarray:
        prefix = f"l{index}.mlp"
        if mlp["kind"] == "dense":
            hidden = clamped_gate(self.linear(f"{prefix}.gate", h), self.linear(f"{prefix}.up", h),
                                  mlp["limit"])
            return self.linear(f"{prefix}.down", self.round(hidden))
        top = mlp["router"]["top"]
        logits = self.linear(f"{prefix}.router", h) + self.w[f"{prefix}.router.b"]
        chosen, weights = choose_experts(logits, top)
        if top < logits.shape[1] and self.margins is not None:
            ordered = -np.sort(-logits, axis=1)
            self.margins = np.minimum(self.margins, ordered[:, top - 1] - ordered[:, top])
        out = np.zeros_like(h)
        for expert in range(mlp["router"]["experts"]):
            rows, place = np.nonzero(chosen == expert)
            if len(rows):
                out[rows] += weights[rows, place][:, None] * \
                    self.small_feed_forward(f"{prefix}.e{expert}", h[rows])
        if mlp.get("shared") is not None:
            out = out + self.small_feed_forward(f"{prefix}.shared", h)
        return out

    def logits(self, tokens) -> np.ndarray:
        return self.forward(tokens).astype(np.float32)

    def hidden_states(self, tokens) -> List[np.ndarray]:
        """The residual after every layer."""
        states: List[np.ndarray] = []
        self.after_layer = lambda layer, x: states.append(x.copy())
        try:
            self.forward(tokens)
        finally:
            self.after_layer = None
        return states

    def forward(self, tokens) -> np.ndarray:
        """Logits ``[T, vocab]`` of one whole sequence from position 0."""
        tokens = np.asarray(tokens, dtype=np.int64)
        positions = np.arange(len(tokens), dtype=np.float64)
        self.margins = np.full(len(tokens), np.inf)
        x = self.w["embed"][tokens]
        pairs = (self.config.get("embedding") or {}).get("bigram")
        if pairs:
            x = x + self.w["bigram"][pair_rows(tokens, pairs["buckets"], pairs["mul_prev"],
                                               pairs["mul_cur"])]
        factor = self.config["residual_mult"]
        kept: dict = {}
        for index, layer in enumerate(self.config["layers"]):
            h = self.round(x)
            if layer["type"] == "attention":
                y = self.attention_mixer(index, layer["mixer"], h, positions, kept)
            elif layer["type"] == "mlstm":
                y = self.lstm_mixer(index, layer["mixer"], h)
            else:
                raise ValueError(f"unknown layer type {layer['type']!r}")
            x = x + factor * rms_norm(y, self.w[f"l{index}.norm1"], self.eps)
            if layer.get("mlp") is not None:
                y = self.feed_forward(index, layer["mlp"], self.round(x))
                x = x + factor * rms_norm(y, self.w[f"l{index}.norm2"], self.eps)
            if self.after_layer is not None:
                self.after_layer(index, x)
        final = self.round(rms_norm(x, self.w["final.norm"], self.eps))
        return self.linear("head", final)

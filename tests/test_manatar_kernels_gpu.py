"""The kernels behind the Manatar mechanisms, one at a time, against the plain functions of
``plain_manatar`` (NumPy, double): the embedding with a table of pairs, the norm behind a sublayer
with bias and cleared buffer, the router over the chosen logits, the clamped gate of a dense
feed-forward, biases with filter, norm, rotation and append of heads with two maps, the difference
of the maps, and the matrix memory (token by token, by chunks on the tensor cores, one decoded
token).  Sizes are ones the models of the other tests do not have.
"""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_manatar as plain
from test_rekasun_kernels_gpu import dev, host, status_word
from test_rorovik_kernels_gpu import DTYPES, as_double, bounds, close, device_tensor, held

pytestmark = pytest.mark.gpu


def batch_of(lengths, slots):
    """Device description of one step: ``(token_request, request_slot, request_start)``."""
    starts = np.concatenate([[0], np.cumsum(lengths)])
    return (dev(np.repeat(np.arange(len(lengths)), lengths), torch.int32), dev(slots, torch.int32),
            dev(starts, torch.int32))


def rounds_of(totals, rng, sizes=(1, 2, 3, 5, 9)):
    """Steps of portions: per step a list of (request, begin, end) until all are fed."""
    done = [0] * len(totals)
    while any(d < t for d, t in zip(done, totals)):
        step = []
        for request in rng.permutation(len(totals)):
            if done[request] < totals[request] and rng.random() < 0.8:
                size = min(int(rng.choice(sizes)), totals[request] - done[request])
                step.append((int(request), done[request], done[request] + size))
                done[request] += size
        if step:
            yield step


# ------------------------------------------------------------------ embedding with pairs

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,buckets,mul_prev,mul_cur", [(40, 11, 3, 7), (36, 1, 5, 9), (520, 97, -13, 2147480000),
                                                            (9216, 30, 37, -11)])
def test_embedding_with_a_table_of_pairs(dtype, width, buckets, mul_prev, mul_cur):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(51)
    vocab, totals, slots = 53, [23, 1, 40], [2, 0, 3]
    table, pairs = held(rng.normal(size=(vocab, width)), dtype), held(rng.normal(size=(buckets + 1, width)), dtype)
    tokens = [rng.integers(0, vocab, n) for n in totals]
    want = [table[t] * 1.5 + pairs[plain.pair_rows(t, buckets, mul_prev, mul_cur)] for t in tokens]
    previous = torch.full((5, 1), 7, dtype=torch.int32, device="cuda")
    status = status_word()
    for step in rounds_of(totals, rng):
        ids = np.concatenate([tokens[r][a:b] for r, a, b in step])
        positions = np.concatenate([np.arange(a, b) for _, a, b in step])
        batch = batch_of([b - a for _, a, b in step], [slots[r] for r, _, _ in step])
        out = torch.full((len(ids), width), float("nan"), device="cuda")
        ops.embed_pairs(dev(table, dtype), dev(pairs, dtype), dev(ids, torch.int32),
                        dev(positions, torch.int32), *batch, previous, out, len(ids), buckets, mul_prev,
                        mul_cur, status, scale=1.5)
        close(as_double(out), np.concatenate([want[r][a:b] for r, a, b in step]), atol=1e-6, rtol=1e-6)
    assert int(status.item()) == 0
    assert previous.flatten().tolist() == [tokens[1][-1], 7, tokens[0][-1], tokens[2][-1], 7]


def test_a_token_outside_the_vocabulary_is_flagged():
    from helix_runtime_b200.ops import library as ops
    out = torch.zeros((3, 16), device="cuda")
    status = status_word()
    ops.embed_pairs(torch.ones((4, 16), device="cuda"), torch.ones((6, 16), device="cuda"),
                    dev([1, 4, 2], torch.int32), dev([0, 1, 2], torch.int32), *batch_of([3], [0]),
                    torch.zeros((1, 1), dtype=torch.int32, device="cuda"), out, 3, 5, 3, 2, status)
    assert int(status.item()) == ops.FLAG_BAD_TOKEN
    assert torch.isnan(out[1]).all() and torch.isfinite(out[[0, 2]]).all()


# --------------------------------------------------------------- norm behind a sublayer

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 75, 1000, 9000])
@pytest.mark.parametrize("with_bias", [True, False])
def test_norm_behind_a_sublayer_with_bias_and_cleared_buffer(dtype, width, with_bias):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(52)
    x, y = rng.normal(size=(6, width)), 3.0 * rng.normal(size=(6, width))
    w, b = 1.0 + 0.3 * rng.normal(size=width), 2.0 * rng.normal(size=width)
    x, y, w, b = (held(v, torch.float32) for v in (x, y, w, b))
    residual, output = device_tensor(x), device_tensor(y)
    rows = torch.full((6, width), float("nan"), dtype=dtype, device="cuda")
    ops.norm_residual_add(residual, output, device_tensor(w), 1e-4, -0.7, 5, cast_out=rows,
                          bias=device_tensor(b) if with_bias else None, clear=True)
    want = x[:5] - 0.7 * plain.rms_norm(y[:5] + (b if with_bias else 0.0), w, 1e-4)
    close(as_double(residual)[:5], want, atol=1e-5, rtol=1e-5)
    np.testing.assert_array_equal(as_double(residual)[5], x[5])
    np.testing.assert_array_equal(as_double(rows)[:5], held(as_double(residual)[:5], dtype))
    assert float(output[:5].abs().sum()) == 0.0
    np.testing.assert_array_equal(as_double(output)[5], y[5])
    cast = torch.full((6, width), float("nan"), dtype=dtype, device="cuda")
    ops.cast_rows(residual, cast, 6)
    np.testing.assert_array_equal(as_double(cast), held(as_double(residual), dtype))


# ---------------------------------------------------------------------- feed-forward

@pytest.mark.parametrize("experts,top", [(3, 1), (7, 7), (45, 5), (130, 32)])
def test_router_over_the_chosen_logits(experts, top):
    """Logits hundreds apart (a softmax over all of them would round the smaller ones to the same
    zero), ties (the lowest index first), a bias that decides the choice."""
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(53)
    z = held(rng.normal(size=(30, experts)) * 3.0, torch.float32)
    z[0] = -200.0 * np.arange(experts)
    z[1] = 0.0
    z[2] *= 100.0
    bias = held(rng.normal(size=experts) * 2.0, torch.float32)
    bias[experts // 2] = 40.0
    for b in (None, bias):
        chosen = torch.empty((30, top), dtype=torch.int32, device="cuda")
        weights = torch.empty((30, top), device="cuda")
        ops.route_top(device_tensor(z), chosen, weights, 30, experts, top, 1.0, chosen_softmax=True,
                      bias=None if b is None else device_tensor(b))
        sums = (z.astype(np.float32) + (0 if b is None else b.astype(np.float32))).astype(np.float64)
        want_chosen, want_weights = plain.choose_experts(sums, top)
        np.testing.assert_array_equal(chosen.cpu().numpy(), want_chosen)
        close(as_double(weights), want_weights, atol=1e-6)


@pytest.mark.parametrize("tokens", [3, 200])
def test_clamped_gate_of_a_dense_feed_forward(tokens):
    """The part alone, as a weight stream and as the product's epilogue, with a clamp that binds for
    most numbers."""
    from helix_runtime_b200.config.spec import PartSpec
    from helix_runtime_b200.parts import build_part
    from test_parts_gpu import context_for
    rng = np.random.default_rng(54)
    width, ff, limit = 136, 264, 0.6
    w = {name: held(rng.normal(size=shape) / math.sqrt(shape[1]) * 1.5, torch.bfloat16)
         for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    x = held(rng.normal(size=(tokens, width)), torch.bfloat16)
    hidden = plain.clamped_gate(x @ w["gate"].T, x @ w["up"].T, limit)
    part = build_part("feed_forward", PartSpec("gated_mlp", {
        "intermediate_size": ff, "activation": "clamped_sigmoid", "limit": limit},
        {name: name for name in w}), width)
    part.bind({name: dev(value, torch.bfloat16) for name, value in w.items()}, torch.bfloat16,
              torch.device("cuda"))
    ctx = context_for(torch.bfloat16, {}, [("a", tokens)], max_positions=256)[0]
    rows = torch.zeros((256, width), dtype=torch.bfloat16, device="cuda")
    rows[:tokens] = dev(x, torch.bfloat16)
    out = torch.zeros((256, width), device="cuda")
    part.forward(ctx, rows, out)
    close(as_double(out)[:tokens], held(hidden, torch.bfloat16) @ w["down"].T, atol=2e-2, rtol=1e-2)


# -------------------------------------------------- heads: bias, filter, norm, rotation, append

def head_case(rng, dtype, heads, kv_heads, dim, vdim, row_dim, taps, rot, totals, slots, maps=2,
              page_size=8, sums=False, with_norm=True, with_bias=True, sizes=(1, 2, 3, 5, 9)):
    from helix_runtime_b200.ops import library as ops
    q_size, k_size, v_size = heads * maps * dim, kv_heads * maps * dim, kv_heads * vdim
    channels = q_size + k_size + v_size
    extra = 16                                         # columns behind the filtered ones
    projected = [held(rng.normal(size=(n, channels)), dtype) for n in totals]
    bias = held(rng.normal(size=channels) * 0.5, torch.float32) if with_bias else np.zeros(channels)
    filters = held(rng.normal(size=(channels, taps)), torch.float32)
    norms = [held(1.0 + 0.3 * rng.normal(size=dim), torch.float32) for _ in range(2)] if with_norm else [None] * 2
    eps, length = 1e-3, max(totals)
    frequency, amplitude = plain.rotary_frequencies(rot, 50.0, {"factor": 3.0, "original": 20, "fast": 4.0,
                                                                "slow": 0.5}) if rot else (np.zeros(1), 1.0)
    angle = np.arange(length)[:, None] * frequency[None, :]
    want = []
    for rows in projected:
        y = plain.causal_filter(rows + bias, filters)
        positions = np.arange(len(rows), dtype=np.float64)

        def prepared(part, weight):
            part = part.reshape(len(rows), -1, dim)
            if weight is not None:
                part = plain.rms_norm(part, weight, eps)
            return plain.rotate_neighbours(part, positions, frequency, amplitude) if rot else part
        want.append((prepared(y[:, :q_size], norms[0]), prepared(y[:, q_size:q_size + k_size], norms[1]),
                     y[:, q_size + k_size:].reshape(len(rows), kv_heads, vdim) if kv_heads else None))
    pages = sum(-(-n // page_size) for n in totals) + 2
    order = rng.permutation(pages)
    tables, cursor = np.full((max(slots) + 1, 20), -1, dtype=np.int32), 0
    for slot, n in zip(slots, totals):
        count = -(-n // page_size)
        tables[slot, :count] = order[cursor:cursor + count]
        cursor += count
    cache = [torch.full((pages, max(kv_heads, 1), page_size * row_dim), float("nan"), dtype=dtype, device="cuda")
             for _ in range(2)]
    state_size = (taps - 1) * channels
    state = torch.zeros((max(slots) + 1, max(state_size + 4 - state_size % 4, 4)), device="cuda")
    status = status_word()
    got_q = [np.full((n, heads * maps, row_dim), np.nan) for n in totals]
    for step in rounds_of(totals, rng, sizes):
        raw = np.concatenate([projected[r][a:b] for r, a, b in step])
        n = len(raw)
        raw = np.concatenate([raw, rng.normal(size=(n, extra))], axis=1)
        positions = np.concatenate([np.arange(a, b) for _, a, b in step])
        batch = batch_of([b - a for _, a, b in step], [slots[r] for r, _, _ in step])
        rows = torch.full((n, heads * maps * row_dim), float("nan"), dtype=dtype, device="cuda")
        stride = -(-(channels + extra) // 8) * 8
        source = torch.zeros((n, stride), dtype=torch.float32 if sums else dtype, device="cuda")
        source[:, :channels + extra] = dev(raw, source.dtype)
        ops.filtered_heads(source, sums, rows, device_tensor(filters),
                           device_tensor(bias) if with_bias else None, state if taps > 1 else None,
                           *(None if w is None else device_tensor(w) for w in norms), eps,
                           device_tensor(np.cos(angle) * amplitude) if rot else None,
                           device_tensor(np.sin(angle) * amplitude) if rot else None, rot,
                           dev(positions, torch.int32), *batch, n, heads, kv_heads, maps, dim, vdim,
                           row_dim, block_tables=dev(tables, torch.int32) if kv_heads else None,
                           k_cache=cache[0] if kv_heads else None, v_cache=cache[1] if kv_heads else None,
                           page_size=page_size, num_pages=pages, status=status)
        flat = as_double(rows).reshape(n, heads * maps, row_dim)
        cursor = 0
        for r, a, b in step:
            got_q[r][a:b] = flat[cursor:cursor + b - a]
            cursor += b - a
    assert int(status.item()) == 0
    limit = bounds(dtype)
    chunk = 16 // cache[0].element_size()
    chunk = chunk if row_dim % chunk == 0 else (4 if chunk > 4 and row_dim % 4 == 0 else 2)
    stored = [as_double(c).reshape(pages, max(kv_heads, 1), row_dim // chunk, page_size, chunk)
              .transpose(0, 1, 3, 2, 4).reshape(pages, max(kv_heads, 1), page_size, row_dim) for c in cache]
    untouched = np.ones((pages, page_size), dtype=bool)
    for request, (slot, n) in enumerate(zip(slots, totals)):
        q, k, v = want[request]
        for unit in range(heads * maps):
            row = np.zeros((n, row_dim))
            part = unit % maps
            row[:, part * dim:(part + 1) * dim] = q[:, unit]
            close(got_q[request][:, unit], row, what=f"request {request} query {unit}", **limit)
        if not kv_heads:
            continue
        for position in range(n):
            page, place = tables[slot, position // page_size], position % page_size
            untouched[page, place] = False
            row = np.zeros((kv_heads, row_dim))
            row[:, :maps * dim] = k[position].reshape(kv_heads, maps * dim)
            close(stored[0][page, :, place], row, what=f"request {request} key {position}", **limit)
            row[:] = 0.0
            row[:, :vdim] = v[position]
            close(stored[1][page, :, place], row, what=f"request {request} value {position}", **limit)
    if kv_heads:
        for part in stored:
            assert np.isnan(part[untouched.nonzero()[0], :, untouched.nonzero()[1]]).all()


# (dtype, sums): pieces of eight channels, pairs, and any sizes, by the sizes below
HEAD_FORMS = [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)]


@pytest.mark.parametrize("dtype,sums", HEAD_FORMS)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,row_dim,rot", [
    (4, 2, 16, 32, 32, 16), (6, 2, 24, 56, 64, 8), (2, 1, 64, 128, 128, 64), (3, 1, 40, 24, 80, 12),
    (5, 5, 8, 8, 16, 4), (2, 2, 10, 6, 32, 4), (3, 1, 9, 7, 32, 4), (2, 1, 150, 90, 320, 150),
    (1, 1, 120, 264, 288, 0)])
def test_heads_in_portions(dtype, sums, heads, kv_heads, dim, vdim, row_dim, rot):
    for seed, taps in enumerate((1, 2, 3, 4, 6)):
        rng = np.random.default_rng(100 * taps + dim)
        head_case(rng, dtype, heads, kv_heads, dim, vdim, row_dim, taps, rot, [31, 1, 17, 6],
                  [1, 4, 0, 2], sums=sums)


@pytest.mark.parametrize("dtype,sums", HEAD_FORMS)
@pytest.mark.parametrize("dim", [32, 10, 9])
def test_heads_without_keys_norm_or_bias(dtype, sums, dim):
    rng = np.random.default_rng(61)
    head_case(rng, dtype, 4, 0, dim, 12, 96, 3, 4, [20, 3, 11], [0, 2, 1], sums=sums)
    head_case(rng, dtype, 4, 2, dim, 12, 96, 3, 4, [20, 3, 11], [0, 2, 1], sums=sums, with_norm=False)
    head_case(rng, dtype, 4, 2, dim, 12, 96, 3, 4, [20, 3, 11], [0, 2, 1], sums=sums, with_bias=False)


@pytest.mark.parametrize("dtype", DTYPES)
def test_heads_in_portions_of_hundreds(dtype):
    """Runs of tokens that cross requests and begin inside portions."""
    rng = np.random.default_rng(62)
    head_case(rng, dtype, 2, 1, 16, 24, 32, 4, 16, [150, 149, 3, 120], [1, 0, 3, 2], sizes=(150, 147, 2))
    head_case(rng, dtype, 2, 1, 16, 24, 32, 4, 16, [159, 159, 1, 158, 157, 159, 150, 159], list(range(8)),
              sizes=(159, 150), page_size=16)


def test_a_position_beyond_the_table_is_flagged():
    from helix_runtime_b200.ops import library as ops
    for dim in (8, 6, 5):
        status = status_word()
        row = torch.zeros((1, 32), dtype=torch.bfloat16, device="cuda")
        ops.filtered_heads(torch.ones((1, 16), dtype=torch.bfloat16, device="cuda"), False, row,
                           torch.ones((2 * dim, 1), device="cuda"), None, None, None, None, 0.0,
                           torch.ones((4, 2), device="cuda"), torch.ones((4, 2), device="cuda"), 4,
                           dev([4], torch.int32), *batch_of([1], [0]), 1, 1, 0, 2, dim, 4, 16,
                           status=status)
        assert int(status.item()) == ops.FLAG_BAD_POSITION


# --------------------------------------------------------------- difference of the maps

@pytest.mark.parametrize("dtype,sums", HEAD_FORMS)
@pytest.mark.parametrize("heads,vdim,row_dim", [(3, 24, 32), (9, 100, 112), (2, 7, 32), (4, 128, 128),
                                                (2, 300, 320)])
def test_difference_of_maps(dtype, sums, heads, vdim, row_dim):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(63)
    tokens, front, lam, diff, eps = 7, 20, 0.43, 0.3, 1e-3
    context = np.full((tokens, 2 * heads, row_dim), np.nan)
    context[:, :, :vdim] = held(rng.normal(size=(tokens, 2 * heads, vdim)), dtype)
    context[0, 1] = context[0, 0] / lam            # a difference near zero: eps decides
    context[:, :, :vdim] = held(context[:, :, :vdim], dtype)
    gate = held(rng.normal(size=(tokens, heads * vdim)) * 3.0, dtype)
    width = front + heads * vdim
    rows = torch.full((tokens, width), 1.0, dtype=torch.float32 if sums else dtype, device="cuda")
    rows[:, front:] = dev(gate, rows.dtype)
    out = torch.full((tokens, heads * vdim), float("nan"), dtype=dtype, device="cuda")
    ops.map_difference(dev(context.reshape(tokens, -1), dtype), rows[:, front:], sums, lam, 1.0 - diff, eps,
                       out, tokens, heads, vdim, row_dim, clear=rows if sums else None)
    a = context[:, :, :vdim].reshape(tokens, heads, 2, vdim)
    want = plain.difference_of_maps(a[:, :, 0], a[:, :, 1], lam, diff, eps).reshape(tokens, -1) * plain.sigmoid(gate)
    close(as_double(out), want, **(dict(atol=2e-4, rtol=2e-4) if dtype == torch.float32 else bounds(dtype)))
    assert not sums or float(rows.abs().sum()) == 0.0


# --------------------------------------------------------------------- matrix memory

class LstmCase:
    """Requests of a matrix memory fed in steps; ``decode``: single tokens take the one-token kernel.
    ``chunks``: the tensor-core form for steps with longer portions."""

    def __init__(self, rng, dtype, heads, dim, vdim, cap, totals, bias=None, gate_gain=1.0):
        self.dtype, self.heads, self.dim, self.vdim, self.cap, self.totals = dtype, heads, dim, vdim, cap, totals
        self.rows = [held(rng.normal(size=(n, 2 * heads * (dim + vdim))), dtype) for n in totals]
        self.gates = [held(rng.normal(size=(n, 2 * heads)) * gate_gain, torch.float32) for n in totals]
        if bias is None:
            bias = np.concatenate([rng.normal(size=heads), np.resize([5.0, 0.5, 9.0], heads)])
        self.bias = held(bias, torch.float32)
        self.norm = held(1.0 + 0.3 * rng.normal(size=heads * vdim), torch.float32)
        self.scale, self.floor, self.eps = dim ** -0.5, 1e-6, 1e-5

    def expected(self, request):
        h, d, e = self.heads, self.dim, self.vdim
        rows, n = self.rows[request], self.totals[request]
        q = rows[:, :h * d].reshape(n, h, d) * self.scale
        k = rows[:, h * d:2 * h * d].reshape(n, h, d)
        v = rows[:, 2 * h * d:2 * h * d + h * e].reshape(n, h, e)
        gate = rows[:, 2 * h * d + h * e:]
        z = self.gates[request] + self.bias
        log_in, log_forget = plain.lstm_gates(z[:, :h], z[:, h:], self.cap)
        out = np.stack([plain.unit_rms(plain.matrix_lstm(q[:, i], k[:, i], v[:, i], log_in[:, i],
                                                         log_forget[:, i], self.floor), self.eps)
                        for i in range(h)], axis=1)
        return out.reshape(n, h * e) * self.norm * plain.sigmoid(gate)

    def run(self, steps, slots, chunks, sums=False, capacity=None):
        from helix_runtime_b200.ops import library as ops
        h, d, e = self.heads, self.dim, self.vdim
        width, dtype = 2 * h * (d + e), self.dtype
        floats = ops.matrix_lstm_state_floats(h, d, e)
        state = torch.full((max(slots) + 2, floats + 3), float("nan"), device="cuda")
        for slot in slots:
            state[slot].zero_()
        got = [np.full((n, h * e), np.nan) for n in self.totals]
        capacity = capacity or max(sum(b - a for _, a, b in step) for step in steps) + 5
        for step in steps:
            lengths = [b - a for _, a, b in step]
            n = sum(lengths)
            one_token = n == len(step)
            raw = np.concatenate([self.rows[r][a:b] for r, a, b in step])
            z = np.concatenate([self.gates[r][a:b] for r, a, b in step])
            batch = batch_of(lengths, [slots[r] for r, _, _ in step])
            o = torch.full((capacity, h * e), float("nan"), device="cuda")
            arrays = torch.full((5, h, capacity), float("nan"), device="cuda")
            out = torch.full((capacity, h * e + 8 - h * e % 8), float("nan"), dtype=dtype, device="cuda")[:, :h * e]
            accumulate = sums and one_token
            if accumulate:
                rows = torch.zeros((n, -(-(width + 2 * h) // 4) * 4), device="cuda")
                rows[:, :width], rows[:, width:width + 2 * h] = device_tensor(raw), device_tensor(z)
                gate_sums = rows[:, width:]
            else:
                rows = torch.zeros((n, -(-width // 8) * 8), dtype=dtype, device="cuda")
                rows[:, :width] = dev(raw, dtype)
                gate_sums = device_tensor(z)
            tail = (n, h, d, e)
            if not one_token:
                ops.matrix_lstm_gates(gate_sums, device_tensor(self.bias), self.cap, arrays[0], arrays[1],
                                      arrays[2], state, batch[2], batch[1], len(step), *tail)
            by_chunks = chunks and not one_token
            if by_chunks:
                scratch = torch.full((ops.state_chunks_scratch(h, capacity),), float("nan"),
                                     dtype=dtype, device="cuda")
                a, b = h * d, 2 * h * d
                ops.state_chunks(rows[:, :a], rows[:, a:b], rows[:, b:b + h * e], arrays[0], arrays[1],
                                 arrays[4], scratch, self.scale, state, o, arrays[3], batch[2], batch[1],
                                 len(step), ops.recurrence_tiles(lengths), h, d, e)
            ops.matrix_lstm(rows, accumulate, device_tensor(self.bias), self.cap,
                            None if one_token else tuple(arrays[:3]), gate_sums if one_token else None,
                            self.scale, self.floor, device_tensor(self.norm), self.eps, state, o, arrays[3],
                            out, *batch[:1], batch[2], batch[1], len(step), *tail, scan=not by_chunks)
            assert not accumulate or float(rows.abs().sum()) == 0.0
            flat, cursor = as_double(out[:n]), 0
            for r, a, b in step:
                got[r][a:b] = flat[cursor:cursor + b - a]
                cursor += b - a
        others = [slot for slot in range(max(slots) + 2) if slot not in slots]
        assert torch.isnan(state[others]).all()
        return got

    def check(self, steps, slots, what, **options):
        got = self.run(list(steps), slots, **options)
        for request in range(len(self.totals)):
            # values of order one, a few of them behind a divisor near its bound
            limit = dict(atol=3e-4, rtol=3e-4) if self.dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
            close(got[request], self.expected(request), what=f"{what} request {request}", **limit)


LSTM_FORMS = [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)]


@pytest.mark.parametrize("dtype,chunks", LSTM_FORMS)
@pytest.mark.parametrize("heads,dim,vdim,cap", [(3, 16, 24, 15.0), (2, 64, 128, 5.0), (1, 200, 104, 8.0),
                                                (5, 8, 8, 2.0), (2, 136, 40, 15.0), (1, 304, 72, 15.0),
                                                (1, 512, 16, 15.0), (9, 40, 264, 15.0)])
def test_matrix_memory_in_portions_and_decoding(dtype, chunks, heads, dim, vdim, cap):
    rng = np.random.default_rng(dim + vdim)
    case = LstmCase(rng, dtype, heads, dim, vdim, cap, [150, 1, 64, 97])
    slots = [2, 0, 4, 1]
    whole = [[(0, 0, 150), (1, 0, 1), (2, 0, 64), (3, 0, 97)]]
    case.check(whole, slots, "whole", chunks=chunks)
    case.check(rounds_of(case.totals, rng, (1, 2, 5, 63, 64, 65)), slots, "portions", chunks=chunks)
    decoded = [[(0, 0, 130), (2, 0, 50)]] + [[(0, 130 + t, 131 + t)] + ([(2, 50 + t, 51 + t)] if t < 14 else [])
                                              for t in range(20)]
    case.totals = [150, 0, 64, 0]
    case.rows[1], case.rows[3] = case.rows[1][:0], case.rows[3][:0]
    case.gates[1], case.gates[3] = case.gates[1][:0], case.gates[3][:0]
    case.check(decoded, slots, "decoded", chunks=chunks, sums=dtype == torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_of_sizes_without_chunks(dtype):
    from helix_runtime_b200.ops import library as ops
    assert not ops.state_chunks_supports(18, 7) and not ops.state_chunks_supports(520, 8)
    rng = np.random.default_rng(71)
    for heads, dim, vdim in ((3, 18, 7), (1, 5, 1), (40, 3, 2)):
        case = LstmCase(rng, dtype, heads, dim, vdim, 4.0, [50, 3])
        case.eps = 0.3      # heads of one or two values: not only their signs
        case.check(rounds_of(case.totals, rng), [1, 0], f"{heads} {dim} {vdim}", chunks=False)


@pytest.mark.parametrize("dtype,chunks", LSTM_FORMS)
def test_a_far_token_that_stands_out(dtype, chunks):
    """A token 300 positions back whose input gate is open wide while all others are nearly shut, in
    a head that hardly forgets and in one that forgets half at every token: the first head still
    answers with its value, the second has lost it."""
    rng = np.random.default_rng(72)
    heads, dim, vdim, total, far = 2, 32, 32, 330, 20
    case = LstmCase(rng, dtype, heads, dim, vdim, 15.0, [total],
                    bias=np.array([-12.0, -12.0, 14.0, 0.0]), gate_gain=0.1)
    case.gates[0][far, :heads] = 30.0
    steps = [[(0, 0, 200)], [(0, 200, 320)]] + [[(0, t, t + 1)] for t in range(320, total)]
    case.check(steps, [0], "far token", chunks=chunks)
    want = case.expected(0)
    value = held(case.rows[0][far, 2 * heads * dim:2 * heads * dim + vdim], dtype)
    shown = want[-1, :vdim] / (case.norm[:vdim] * plain.sigmoid(case.rows[0][-1, -2 * vdim:-vdim]))
    assert abs(np.corrcoef(shown, value)[0, 1]) > 0.99


@pytest.mark.parametrize("dtype,chunks", LSTM_FORMS)
def test_gates_that_hardly_forget_over_thousands_of_tokens(dtype, chunks):
    """Forget gates of 1 - 3e-7 to 1 - 1e-3 over 3,000 tokens: neither the running maximum's rounding
    nor the decays' may add up."""
    rng = np.random.default_rng(73)
    case = LstmCase(rng, dtype, 3, 16, 16, 15.0, [3000], bias=np.array([0.5, 0.0, -1.0, 40.0, 12.0, 7.0]),
                    gate_gain=0.3)
    case.check([[(0, 0, 1500)], [(0, 1500, 1502)], [(0, 1502, 2999)], [(0, 2999, 3000)]], [0], "slow", chunks=chunks)


def test_chunks_agree_with_the_scan_closely():
    """Both forms from the same bfloat16 rows, compared in float32 before the norm: the chunks carry
    about 16 bits of every factor."""
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(74)
    heads, dim, vdim, n = 2, 72, 88, 203
    case = LstmCase(rng, torch.bfloat16, heads, dim, vdim, 15.0, [n])
    rows = dev(case.rows[0], torch.bfloat16)
    batch = batch_of([n], [0])
    results = []
    for chunks in (False, True):
        state = torch.zeros((1, ops.matrix_lstm_state_floats(heads, dim, vdim)), device="cuda")
        arrays, o = torch.zeros((5, heads, n), device="cuda"), torch.zeros((n, heads * vdim), device="cuda")
        out = torch.zeros((n, heads * vdim), dtype=torch.bfloat16, device="cuda")
        ops.matrix_lstm_gates(device_tensor(case.gates[0]), device_tensor(case.bias), 15.0, arrays[0], arrays[1],
                              arrays[2], state, batch[2], batch[1], 1, n, heads, dim, vdim)
        if chunks:
            a, b = heads * dim, 2 * heads * dim
            scratch = torch.zeros(ops.state_chunks_scratch(heads, n), dtype=torch.bfloat16, device="cuda")
            ops.state_chunks(rows[:, :a], rows[:, a:b], rows[:, b:b + heads * vdim], arrays[0], arrays[1],
                             arrays[4], scratch, case.scale, state, o, arrays[3], batch[2], batch[1], 1,
                             ops.recurrence_tiles([n]), heads, dim, vdim)
        else:
            ops.matrix_lstm(rows, False, device_tensor(case.bias), 15.0, tuple(arrays[:3]), None, case.scale,
                            1e-6, device_tensor(case.norm), 1e-5, state, o, arrays[3], out, batch[0], batch[2],
                            batch[1], 1, n, heads, dim, vdim)
        results.append((as_double(o), as_double(arrays[3]), as_double(state)))
    for got, want, what in zip(results[1], results[0], ("output", "weights", "state")):
        close(got, want, atol=3e-5 * np.abs(want).max(), what=what)

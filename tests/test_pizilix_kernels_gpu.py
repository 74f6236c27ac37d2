"""The kernels behind the Pizilix mechanisms, one at a time, against the plain functions of
``plain_pizilix`` (NumPy, double): the attention kernels with chunks, levels and a constant sink
(CUDA cores, the streaming kernel, the ``mma.sync`` kernel with a head or a token's heads per
tile, the tcgen05 kernel), the rotation and cache append with values that are the keys (on their
own and as the product's epilogue), the filter with a bias on its inputs, the block-diagonal gates
and the scan (token by token and by tiles of tokens), the one-kernel step, and products whose
sums run into a level.  Sizes are ones the models of the other tests do not have.
"""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_pizilix as plain
from test_rekasun_kernels_gpu import dev, host, status_word, to_cache_layout
from test_rorovik_kernels_gpu import (DTYPES, KERNELS, as_double, bounds, close, device_tensor, held,
                                      sizes_for)

pytestmark = pytest.mark.gpu


# --------------------------------------------------- attention with chunks, levels and a sink

def attention_case(rng, dtype, kernel, heads, kv_heads, head_dim, page_size, context, new, chunk,
                   cap, sink=True, dominant=None, scale=None, split_keys=32):
    """One request with ``context`` cached keys and ``new`` query tokens through one kernel.
    ``dominant=(row, key)`` scales the key at that position along that row's query.  Pages of
    chunks that have ended are taken out of the block table, as the cache manager does."""
    from helix_runtime_b200.ops import library as ops
    total = context + new
    keys = held(rng.normal(size=(total, kv_heads, head_dim)), dtype)
    values = held(rng.normal(size=(total, kv_heads, head_dim)), dtype)
    queries = held(rng.normal(size=(new, heads, head_dim)), dtype)
    share = heads // kv_heads
    if dominant is not None:
        row, position = dominant
        for kv in range(kv_heads):
            direction = queries[row, kv * share]
            keys[position, kv] = held(direction / np.linalg.norm(direction) * 60.0, dtype)
            queries[row, kv * share:(kv + 1) * share] = direction
    pages = -(-total // page_size)
    num_pages = pages + 3
    order = rng.permutation(num_pages)
    tables = np.full((2, pages + 1), -1, dtype=np.int32)
    k_cache = np.full((num_pages, kv_heads, page_size, head_dim), np.nan, dtype=np.float32)
    v_cache = np.full_like(k_cache, np.nan)
    first_seen = context // chunk * chunk if chunk else 0
    for p in range(pages):
        lo, hi = p * page_size, min((p + 1) * page_size, total)
        if hi <= first_seen:
            continue                                    # given back: nobody reads it again
        tables[1, p] = order[p]
        k_cache[order[p], :, :hi - lo] = keys[lo:hi].transpose(1, 0, 2)
        v_cache[order[p], :, :hi - lo] = values[lo:hi].transpose(1, 0, 2)
    out = torch.full((new, heads * head_dim), float("nan"), dtype=dtype, device="cuda")
    status = status_word()
    scale = 1.3 / math.sqrt(head_dim) if scale is None else scale
    common = (dev(queries.reshape(new, heads * head_dim), dtype),
              dev(to_cache_layout(k_cache, dtype), dtype), dev(to_cache_layout(v_cache, dtype), dtype))
    options = dict(sinks=device_tensor(np.zeros(heads)) if sink else None, chunk=chunk or 0,
                   softcap=cap or 0.0)
    starts, slots = dev([0, new], torch.int32), dev([1], torch.int32)
    if kernel in ("mma", "packed", "tcgen05"):
        ops.prefill_attention(*common, starts, dev([context], torch.int32), slots,
                              dev(tables, torch.int32), out, 1, new, heads, kv_heads, head_dim,
                              page_size, num_pages, scale, 1, status,
                              tensor_memory=kernel == "tcgen05", packed=kernel == "packed", **options)
    else:
        longest = min(total, chunk) if chunk else total
        ops.paged_attention(*common, dev(np.arange(context, total), torch.int32),
                            dev(np.zeros(new), torch.int32), slots, dev(tables, torch.int32), out,
                            None, new, heads, kv_heads, head_dim, page_size, num_pages, 0, scale,
                            split_keys, max(1, -(-longest // split_keys)), status, group_heads=kernel == "grouped", **options)
    assert int(status.item()) == 0
    padded = np.concatenate([np.zeros((context, heads, head_dim)), queries])
    expected = plain.chunked_attention(padded, keys, values, scale, cap, chunk, sink)[context:]
    return host(out).reshape(new, heads, head_dim), expected, values


@pytest.mark.parametrize("dtype,kernel", KERNELS)
@pytest.mark.parametrize("chunk", [None, 1, 19, 64, 70, 256])
@pytest.mark.parametrize("cap", [None, 2.0])
def test_chunks_and_levels_in_portions_and_decoding(dtype, kernel, chunk, cap):
    rng = np.random.default_rng(27)
    heads, kv_heads = {"packed": (6, 1), "grouped": (14, 2)}.get(kernel, (6, 2))
    for context, new in [(0, 150), (37, 90), (63, 1), (64, 1), (139, 1), (140, 1), (210, 17),
                         (15, 1), (0, 1), (100, 23), (250, 300)]:
        if kernel == "tcgen05" and new == 1:
            continue
        got, want, _ = attention_case(rng, dtype, kernel, heads, kv_heads, *sizes_for(kernel),
                                      context, new, chunk, cap)
        close(got, want, what=f"chunk {chunk} context {context} new {new}", **bounds(dtype))


@pytest.mark.parametrize("dtype,kernel", KERNELS)
def test_scores_far_beyond_and_far_below_their_level(dtype, kernel):
    """Scores of a hundred under a level of 8, of a tenth under a level of 50 (where the level
    hardly shows), and around a level of 3."""
    rng = np.random.default_rng(28)
    head_dim, page = sizes_for(kernel)
    for scale, cap in ((30.0, 8.0), (0.02, 50.0), (1.0, 3.0), (0.3, 1.0)):
        for context, new in ((40, 1), (10, 50)):
            if kernel == "tcgen05" and new == 1:
                continue
            got, want, _ = attention_case(rng, dtype, kernel, 4, 1, head_dim, page, context, new,
                                          None, cap, scale=scale / math.sqrt(head_dim))
            close(got, want, what=f"scale {scale} cap {cap} new {new}", **bounds(dtype))


@pytest.mark.parametrize("dtype,kernel", KERNELS)
def test_one_more_in_the_denominator(dtype, kernel):
    """A position that sees itself alone keeps e^s / (1 + e^s) of its value."""
    rng = np.random.default_rng(29)
    head_dim, page = sizes_for(kernel)
    new = 1 if kernel != "tcgen05" else 40
    for sink in (True, False):
        got, want, values = attention_case(rng, dtype, kernel, 4, 1, head_dim, page, 0, new, 1, None,
                                           sink=sink)
        close(got, want, what=f"sink {sink}", **bounds(dtype))
        assert (np.abs(got - values[:, :1]).max() < 2e-2) == (not sink)


@pytest.mark.parametrize("dtype,kernel", KERNELS)
@pytest.mark.parametrize("new", [1, 80])
def test_a_key_at_a_chunks_edge(dtype, kernel, new):
    """One key is scaled so that it takes nearly all the weight of the last query: the first
    position of the query's chunk is found, the last of the chunk before is not."""
    if kernel == "tcgen05" and new == 1:
        pytest.skip("single tokens are not the tcgen05 kernel's")
    rng = np.random.default_rng(30)
    for chunk, total in ((48, 300), (100, 299), (37, 149), (64, 192), (64, 193)):
        start = (total - 1) // chunk * chunk
        for key in sorted({start, start - 1, start + 1, total - 1} & set(range(total))):
            got, want, values = attention_case(rng, dtype, kernel, 4, 1, sizes_for(kernel)[0], 16,
                                               total - new, new, chunk, 60.0,
                                               dominant=(new - 1, key))
            close(got, want, what=f"chunk {chunk} key {key}", **bounds(dtype))
            distance = float(np.abs(got[-1] - values[key, 0][None, :]).max())
            assert (distance < 3e-2) == (key >= start), f"chunk {chunk} key {key}: {distance}"


def test_a_far_key_among_hundreds_of_its_chunk():
    rng = np.random.default_rng(31)
    for dtype, kernel in KERNELS:
        for new in (1, 40):
            if kernel == "tcgen05" and new == 1:
                continue
            got, want, values = attention_case(rng, dtype, kernel, 4, 1, sizes_for(kernel)[0], 16,
                                               1020 - new, new, 600, 100.0, dominant=(new - 1, 603))
            close(got, want, what=f"{kernel} new {new}", **bounds(dtype))
            assert np.abs(got[-1] - values[603, 0][None, :]).max() < 3e-2


@pytest.mark.parametrize("heads,kv_heads", [(5, 1), (8, 4), (12, 3), (4, 4), (9, 1)])
@pytest.mark.parametrize("chunk", [0, 300])
def test_decoding_requests_of_very_different_lengths_in_groups_of_heads(heads, kv_heads, chunk):
    """One token of each of twelve requests: rows are cut between warps anywhere."""
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(heads + chunk)
    dtype, head_dim, page_size, cap = torch.bfloat16, 64, 16, 3.0
    positions = np.array([0, 1, 15, 16, 31, 299, 300, 301, 640, 1499, 7, 900])
    count = len(positions)
    pages = [int(p) // page_size + 1 for p in positions]
    num_pages = sum(pages) + 2
    order = list(rng.permutation(num_pages))
    tables = np.full((count, max(pages)), -1, dtype=np.int32)
    k_cache = np.full((num_pages, kv_heads, page_size, head_dim), np.nan, dtype=np.float32)
    v_cache = np.full_like(k_cache, np.nan)
    queries = held(rng.normal(size=(count, heads, head_dim)), dtype)
    want, scale = [], 1.5 / math.sqrt(head_dim)
    for request, position in enumerate(positions):
        keys, values = (held(rng.normal(size=(position + 1, kv_heads, head_dim)), dtype)
                        for _ in range(2))
        for p in range(pages[request]):
            lo, hi = p * page_size, min((p + 1) * page_size, position + 1)
            if chunk and hi <= position // chunk * chunk:
                continue
            page = tables[request, p] = order.pop()
            k_cache[page, :, :hi - lo] = keys[lo:hi].transpose(1, 0, 2)
            v_cache[page, :, :hi - lo] = values[lo:hi].transpose(1, 0, 2)
        first = position // chunk * chunk if chunk else 0
        padded = np.concatenate([np.zeros((position - first, heads, head_dim)),
                                 queries[request:request + 1]])
        want.append(plain.chunked_attention(padded, keys[first:], values[first:], scale, cap,
                                            None)[-1])
    out = torch.full((count, heads * head_dim), float("nan"), dtype=dtype, device="cuda")
    arrivals = torch.zeros(count * heads, dtype=torch.int32, device="cuda")
    status = status_word()
    for repeat in range(2):       # the second call finds the counters as the first left them
        ops.paged_attention(dev(queries.reshape(count, -1), dtype),
                            dev(to_cache_layout(k_cache, dtype), dtype),
                            dev(to_cache_layout(v_cache, dtype), dtype),
                            dev(positions, torch.int32), dev(np.arange(count), torch.int32),
                            dev(np.arange(count), torch.int32), dev(tables, torch.int32), out, None,
                            count, heads, kv_heads, head_dim, page_size, num_pages, 0, scale, 32, 48,
                            status, arrivals=arrivals, sinks=device_tensor(np.zeros(heads)),
                            chunk=chunk, softcap=cap, group_heads=True)
        assert int(status.item()) == 0 and not arrivals.any()
        close(host(out).reshape(count, heads, head_dim), np.stack(want), what="decoded",
              **bounds(dtype))


# ------------------------------------------------------------ rotation, values from the keys

def rotation_tables(dims, positions=512):
    frequencies, amplitude = plain.rotary_frequencies(
        dims, 1000.0, {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0})
    angle = np.arange(positions)[:, None] * frequencies[None, :]
    return (frequencies, amplitude, device_tensor(np.cos(angle) * amplitude),
            device_tensor(np.sin(angle) * amplitude))


def check_pages(cache, want, positions, tables, page_size, what, atol, rtol):
    """``cache`` in the kernels' order ``[page, head, dim / c, slot, c]``."""
    for token, position in enumerate(positions):
        page, slot = tables[position // page_size], position % page_size
        got = cache[page, :, :, slot].reshape(cache.shape[1], -1)
        close(got, want[token], atol, rtol, f"{what} of token {token}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,dims", [(5, 1, 32, 8), (4, 2, 48, 48), (3, 3, 10, 4),
                                                     (2, 1, 64, 12), (2, 2, 16, 0)])
@pytest.mark.parametrize("from_sums", [False, True])
def test_rotation_and_append_with_values_from_the_keys(dtype, heads, kv_heads, dim, dims, from_sums):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(dim)
    tokens, page_size, pages = 11, 8, 9
    positions = np.array([0, 1, 7, 8, 9, 30, 31, 32, 33, 40, 63])
    width = (heads + kv_heads) * dim
    rows = held(rng.normal(size=(tokens, width)), dtype)
    frequencies, amplitude, cos, sin = rotation_tables(max(dims, 2))
    q = rows[:, :heads * dim].reshape(tokens, heads, dim)
    k = rows[:, heads * dim:].reshape(tokens, kv_heads, dim)
    turn = lambda x: x if dims == 0 else plain.rotate_neighbours(x, positions, frequencies, amplitude)
    tables = np.full((3, 8), -1, dtype=np.int32)
    tables[2] = rng.permutation(pages)[:8]
    chunk = 16 // (4 if dtype == torch.float32 else 2)
    chunk = chunk if dim % chunk == 0 else (4 if dim % 4 == 0 and dtype != torch.float32 else 2)
    caches = [torch.full((pages, kv_heads, dim // chunk, page_size, chunk), float("nan"), dtype=dtype,
                         device="cuda") for _ in range(2)]
    buffer = torch.full((tokens, width), float("nan"), dtype=dtype, device="cuda")
    sums = None
    if from_sums:
        sums = torch.zeros((tokens, -(-width // 4) * 4), dtype=torch.float32, device="cuda")
        sums[:, :width] = device_tensor(rows)
    else:
        buffer.copy_(device_tensor(rows, dtype))
    status = status_word()
    ops.rope_append(buffer, dev(positions, torch.int32), dev(np.zeros(tokens), torch.int32),
                    dev([2], torch.int32), dev(tables, torch.int32), caches[0], caches[1], cos, sin,
                    tokens, heads, kv_heads, dim, dims, 0, page_size, pages, status, accum=sums,
                    shared_values=True)
    assert int(status.item()) == 0
    tolerance = (1e-5, 1e-5) if dtype == torch.float32 else (1e-2, 8e-3)
    close(as_double(buffer)[:, :heads * dim].reshape(tokens, heads, dim), turn(q), *tolerance, "queries")
    check_pages(as_double(caches[0]), turn(k), positions, tables[2], page_size, "key", *tolerance)
    check_pages(as_double(caches[1]), k, positions, tables[2], page_size, "value", 0.0, 0.0)
    if from_sums:
        assert not sums[:, :width].any()


@pytest.mark.parametrize("heads,kv_heads,dim,dims,tokens", [(3, 1, 48, 16, 70), (4, 2, 64, 24, 300),
                                                            (2, 2, 32, 32, 129)])
def test_rotation_as_the_products_epilogue_with_values_from_the_keys(heads, kv_heads, dim, dims, tokens):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(tokens)
    depth, page_size = 96, 16
    positions = np.arange(5, 5 + tokens)
    pages = -(-(5 + tokens) // page_size) + 1
    width = (heads + kv_heads) * dim
    x = held(rng.normal(size=(tokens, depth)), torch.bfloat16)
    w = held(rng.normal(size=(width, depth)) / math.sqrt(depth), torch.bfloat16)
    rows = plain.to_bfloat16(x @ w.T)
    frequencies, amplitude, cos, sin = rotation_tables(dims)
    tables = np.full((1, pages), -1, dtype=np.int32)
    tables[0] = rng.permutation(pages)
    q = rows[:, :heads * dim].reshape(tokens, heads, dim)
    k = rows[:, heads * dim:].reshape(tokens, kv_heads, dim)
    for tiled in (False, True):
        weight = device_tensor(w, torch.bfloat16)
        held_weight = ops.tile_weights(weight) if tiled else weight
        caches = [torch.full((pages, kv_heads, dim // 8, page_size, 8), float("nan"),
                             dtype=torch.bfloat16, device="cuda") for _ in range(2)]
        out = torch.full((tokens, width), float("nan"), dtype=torch.bfloat16, device="cuda")
        status = status_word()
        ops.gemm_tc_rope_append(device_tensor(x, torch.bfloat16), held_weight, out, tokens,
                                dev(positions, torch.int32), dev(np.zeros(tokens), torch.int32),
                                dev([0], torch.int32), dev(tables, torch.int32), caches[0], caches[1],
                                cos, sin, heads, kv_heads, dim, dims, page_size, pages, status,
                                weight_shape=(width, depth), shared_values=True)
        assert int(status.item()) == 0
        tolerance = (3e-2, 8e-3)
        close(as_double(out)[:, :heads * dim].reshape(tokens, heads, dim),
              plain.rotate_neighbours(q, positions, frequencies, amplitude), *tolerance, "queries")
        check_pages(as_double(caches[0]), plain.rotate_neighbours(k, positions, frequencies, amplitude),
                    positions, tables[0], page_size, "key", *tolerance)
        check_pages(as_double(caches[1]), k, positions, tables[0], page_size, "value", *tolerance)


# -------------------------------------------------------------------- the filter's input bias

def cut(total, portions):
    """Token counts of successive portions of a sequence of ``total`` tokens."""
    sizes, cursor, index = [], 0, 0
    while cursor < total:
        sizes.append(min(portions[index % len(portions)], total - cursor))
        cursor += sizes[-1]
        index += 1
    return sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(24, 4), (40, 1), (13, 3), (264, 2), (16, 6)])
@pytest.mark.parametrize("from_sums", [False, True])
def test_filter_with_a_bias_on_its_inputs(dtype, channels, taps, from_sums):
    """Two requests in portions of changing size; the zeros in front of a sequence get no bias."""
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(channels + taps)
    lengths = (37, 300)
    inputs = [held(rng.normal(size=(length, channels)), dtype) for length in lengths]
    in_bias, bias = (held(rng.normal(size=channels), torch.float32) for _ in range(2))
    weights = held(rng.normal(size=(channels, taps)), torch.float32)
    want = [plain.causal_filter_bias(x + in_bias, weights, bias) for x in inputs]
    got = [np.zeros((0, channels)) for _ in lengths]
    state = torch.zeros((4, max(1, (taps - 1) * channels)), dtype=torch.float32, device="cuda")
    slots = [3, 1]
    plans = [cut(lengths[0], (2, 5, 1)), cut(lengths[1], (64, 3, 1, 90))]
    cursors = [0, 0]
    for turn in range(max(len(plan) for plan in plans)):
        batch = [(r, plans[r][turn]) for r in range(2) if turn < len(plans[r])]
        starts = np.cumsum([0] + [size for _, size in batch])
        n = int(starts[-1])
        rows = np.concatenate([inputs[r][cursors[r]:cursors[r] + size] for r, size in batch])
        wide = -(-channels // 8) * 8 + 8
        raw = torch.zeros((n, wide), dtype=torch.float32 if from_sums else dtype, device="cuda")
        raw[:, 8:8 + channels] = device_tensor(rows, raw.dtype)
        out = torch.full((n, wide), float("nan"), dtype=dtype, device="cuda")[:, :channels]
        ops.causal_filter(raw[:, 8:8 + channels], out, device_tensor(weights), device_tensor(bias),
                          state if taps > 1 else None, n, False,
                          dev(np.repeat(np.arange(len(batch)), [s for _, s in batch]), torch.int32),
                          dev([slots[r] for r, _ in batch], torch.int32), dev(starts, torch.int32),
                          in_bias=device_tensor(in_bias), sums=from_sums)
        for index, (r, size) in enumerate(batch):
            got[r] = np.concatenate([got[r], as_double(out)[starts[index]:starts[index + 1]]])
            cursors[r] += size
    tolerance = (1e-5, 1e-5) if dtype == torch.float32 else (1e-2, 8e-3)
    for r in range(2):
        close(got[r], want[r], *tolerance, f"request {r}")


# ---------------------------------------------------------------------- gates and recurrence

def recurrence_case(rng, dtype, tokens, blocks, size):
    channels = blocks * size
    case = {
        "u": held(rng.normal(size=(tokens, channels)), dtype),
        "y": held(rng.normal(size=(tokens, channels)) * 1.5, dtype),
        "r": held(rng.normal(size=(blocks, size, size)) * 1.5 / math.sqrt(size), dtype),
        "i": held(rng.normal(size=(blocks, size, size)) * 1.5 / math.sqrt(size), dtype),
        "br": held(rng.normal(size=channels) * 0.5, torch.float32),
        "bi": held(rng.normal(size=channels) * 0.5, torch.float32),
        "by": held(rng.normal(size=channels) * 0.5, torch.float32),
        "lam": rng.uniform(-9.0, 1.0, size=channels),
    }
    case["rate"] = held(8.0 * plain.softplus(case["lam"]), torch.float32)
    case["r_gate"] = plain.sigmoid(plain.block_products(case["u"], case["r"],
                                                        case["br"].reshape(blocks, size)))
    case["i_gate"] = plain.sigmoid(plain.block_products(case["u"], case["i"],
                                                        case["bi"].reshape(blocks, size)))
    return case


def gate_arguments(case, dtype):
    """u in rows of a multiple of eight numbers, the stacked matrices and the vectors."""
    tokens, channels = case["u"].shape
    u = torch.zeros((tokens, -(-channels // 8) * 8), dtype=dtype, device="cuda")
    u[:, :channels] = device_tensor(case["u"], dtype)
    weights = device_tensor(np.stack([case["r"], case["i"]], axis=1), dtype)
    return (u, weights, device_tensor(case["br"]), device_tensor(case["bi"]),
            device_tensor(case["rate"]))


BLOCKS = [(3, 8), (2, 15), (5, 24), (1, 40), (2, 72), (3, 128), (2, 200), (1, 256), (4, 1), (1, 344)]


@pytest.mark.parametrize("dtype,tiled", [(torch.float32, False), (torch.bfloat16, False),
                                         (torch.bfloat16, True)])
@pytest.mark.parametrize("blocks,size", BLOCKS)
def test_block_diagonal_gates(dtype, tiled, blocks, size):
    from helix_runtime_b200.ops import library as ops
    if tiled and not ops.gated_recurrence_supports(size):
        pytest.skip("blocks of a multiple of 8 channels")
    rng = np.random.default_rng(blocks * 1000 + size)
    for tokens in (1, 70, 300):
        case = recurrence_case(rng, dtype, tokens, blocks, size)
        decay, push = (torch.full((tokens, blocks * size), float("nan"), device="cuda")
                       for _ in range(2))
        if tiled:
            # three requests, one of them a single token
            starts = [0, tokens] if tokens == 1 else [0, 1, tokens - 5, tokens]
            count = len(starts) - 1
            joined = torch.full((tokens // 64 + count, 2 * blocks * size), float("nan"), device="cuda")
            before = torch.full((count, blocks * size), float("nan"), device="cuda")
            state = torch.randn((4, blocks * size + 3), device="cuda")
            slots = dev([3, 1, 0][:count], torch.int32)
            tiles = ops.recurrence_tiles(np.diff(starts))
            ops.block_gates_tiled(*gate_arguments(case, dtype), decay, push, joined, state, before,
                                  dev(starts, torch.int32), slots, count, tiles)
            assert torch.equal(before, state[slots.long(), :blocks * size])
        else:
            ops.block_gates(*gate_arguments(case, dtype), decay, push, tokens)
        log_a = -case["r_gate"] * case["rate"]
        # a decay close to one keeps its digits: the error is relative to a - 1
        close(as_double(decay), np.expm1(log_a), 1e-9, 2e-5, f"{tokens} tokens: a - 1")
        close(as_double(push), np.sqrt(-np.expm1(2.0 * log_a)) * case["i_gate"] * case["u"], 1e-7,
              4e-5, f"{tokens} tokens: push")


def run_scan(case, dtype, sizes, slot, state, from_sums, form):
    """The recurrence over one sequence in portions; ``form``: gates and scan, the same by
    tiles, or the one-kernel step (portions of one token)."""
    from helix_runtime_b200.ops import library as ops
    u, weights, br, bi, rate = gate_arguments(case, dtype)
    channels = case["by"].size
    rows, cursor = [], 0
    for count in sizes:
        part = slice(cursor, cursor + count)
        cursor += count
        if from_sums:
            y = torch.zeros((count + 1, 2 * channels), device="cuda")
            y[:count, :channels] = device_tensor(case["y"][part])
            y[:, channels:] = 3.0
        else:
            y = device_tensor(case["y"][part], dtype)
        out = torch.full((count, channels), float("nan"), dtype=dtype, device="cuda")
        slots = dev([slot], torch.int32)
        if form == "step":
            ops.gated_recurrence_step(u[part].contiguous(), weights, br, bi, rate, y,
                                      device_tensor(case["by"]), state, out, 1,
                                      dev([0], torch.int32), slots, sums=from_sums)
        else:
            decay, push = (torch.empty((count, channels), device="cuda") for _ in range(2))
            gates = (u[part].contiguous(), weights, br, bi, rate, decay, push)
            starts = dev([0, count], torch.int32)
            if form == "tiled":
                tiles = ops.recurrence_tiles([count])
                joined = torch.full((tiles, 2 * channels), float("nan"), device="cuda")
                before = torch.full((1, channels), float("nan"), device="cuda")
                ops.block_gates_tiled(*gates, joined, state, before, starts, slots, 1, tiles)
                ops.gated_scan_tiled(decay, push, joined, before, y, device_tensor(case["by"]), state,
                                     out, starts, slots, 1, tiles, sums=from_sums)
            else:
                ops.block_gates(*gates, count)
                ops.gated_scan(decay, push, y, device_tensor(case["by"]), state, out, starts, slots,
                               1, sums=from_sums)
        if from_sums:       # the rows that were read are clear, the row behind them is not touched
            assert not y[:count].any() and bool((y[count, channels:] == 3.0).all())
        rows.append(as_double(out))
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("blocks,size", [(3, 8), (2, 15), (1, 72), (2, 40)])
@pytest.mark.parametrize("from_sums", [False, True])
def test_recurrence_in_portions(dtype, blocks, size, from_sums):
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(size)
    total = 710
    case = recurrence_case(rng, dtype, total, blocks, size)
    states = plain.gated_linear_recurrence(case["u"], case["r_gate"], case["i_gate"], case["lam"])
    want = states * plain.gelu_tanh(case["y"] + case["by"])
    tolerance = (2e-5, 2e-5) if dtype == torch.float32 else (1e-2, 8e-3)
    forms = [("scan", (total,)), ("scan", (64, 2, 3, 61, 580)), ("scan", (1,) * 4 + (2,) * 353),
             ("scan", (63, 65, 7, 575))]
    if dtype == torch.bfloat16 and ops.gated_recurrence_supports(size):
        forms += [("tiled", sizes) for _, sizes in forms] + [("step", (1,) * total)]
    for form, sizes in forms:
        state = torch.zeros((3, blocks * size + 5), device="cuda")
        state[0] = state[2] = 7.0
        got = run_scan(case, dtype, sizes, 1, state, from_sums, form)
        close(got, want, *tolerance, f"{form} {sizes[:4]}")
        close(as_double(state)[1, :blocks * size], states[-1], 2e-5, 4e-5, f"{form}: state")
        assert bool((state[[0, 2]] == 7.0).all()) and not state[1, blocks * size:].any()


@pytest.mark.parametrize("tokens", [1, 3, 8, 9, 16, 20, 33, 64, 70, 129])
@pytest.mark.parametrize("blocks,size", [(2, 40), (3, 8), (1, 264)])
def test_one_kernel_step_of_many_requests(tokens, blocks, size):
    """Every request with its own state and slot, against gates and one step in double."""
    from helix_runtime_b200.ops import library as ops
    rng = np.random.default_rng(tokens)
    case = recurrence_case(rng, torch.bfloat16, tokens, blocks, size)
    channels = blocks * size
    slots = rng.permutation(tokens + 2)[:tokens]
    before = held(rng.normal(size=(tokens + 2, channels)), torch.float32)
    for from_sums in (False, True):
        state = device_tensor(before)
        y = device_tensor(case["y"], torch.bfloat16)
        if from_sums:
            y = torch.cat([device_tensor(case["y"]), torch.ones((tokens, channels), device="cuda")], 1)
        out = torch.full((tokens, channels), float("nan"), dtype=torch.bfloat16, device="cuda")
        ops.gated_recurrence_step(*gate_arguments(case, torch.bfloat16), y.contiguous(),
                                  device_tensor(case["by"]), state, out, tokens,
                                  dev(np.arange(tokens), torch.int32), dev(slots, torch.int32),
                                  sums=from_sums)
        log_a = -case["r_gate"] * case["rate"]
        after = np.exp(log_a) * before[slots] \
            + np.sqrt(-np.expm1(2.0 * log_a)) * case["i_gate"] * case["u"]
        close(as_double(out), after * plain.gelu_tanh(case["y"] + case["by"]), 1e-2, 8e-3, "output")
        close(as_double(state)[slots], after, 2e-5, 2e-5, "state")
        others = np.setdiff1d(np.arange(tokens + 2), slots)
        assert (as_double(state)[others] == before[others]).all()


def test_slow_channels_over_thousands_of_tokens_in_float32():
    """Channels that keep 0.9999 of their state per token and more: the float32 engine's error
    does not grow with the position."""
    rng = np.random.default_rng(40)
    tokens, channels = 4000, 64
    case = recurrence_case(rng, torch.float32, tokens, 1, channels)
    case["lam"] = np.linspace(-14.0, -9.0, channels)
    case["rate"] = held(8.0 * plain.softplus(case["lam"]), torch.float32)
    # the plain recurrence with the decays the device holds
    log_a = -case["r_gate"] * case["rate"]
    state, want = np.zeros(channels), np.zeros((tokens, channels))
    for t in range(tokens):
        state = np.exp(log_a[t]) * state \
            + np.sqrt(-np.expm1(2.0 * log_a[t])) * case["i_gate"][t] * case["u"][t]
        want[t] = state
    want *= plain.gelu_tanh(case["y"] + case["by"])
    held_state = torch.zeros((1, channels), device="cuda")
    got = run_scan(case, torch.float32, (2100, 1900), 0, held_state, False, "scan")
    close(got, want, 3e-6, 3e-6, "4,000 tokens")


# ------------------------------------------------------------------ products with a level

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 5, 20, 60, 129, 300])
def test_products_whose_sums_run_into_a_level(dtype, tokens):
    from helix_runtime_b200.config.spec import PartSpec  # noqa: F401
    from helix_runtime_b200.ops import library as ops
    from helix_runtime_b200.parts.linear import Weight, project
    rng = np.random.default_rng(tokens)
    features, depth, cap = 203, 96, 4.0
    x = held(rng.normal(size=(tokens, depth)), dtype)
    w = held(rng.normal(size=(features, depth)) * 0.6, dtype)
    out = torch.full((tokens, features + 5), float("nan"), device="cuda")
    project(device_tensor(x, dtype), Weight(device_tensor(w, dtype)), out, tokens, ops.EPI_STORE_F32,
            status_word(), softcap=cap)
    want = plain.softcap(x @ w.T, cap)
    assert np.abs(want).max() > 3.9
    close(as_double(out)[:, :features], want, 2e-5, 2e-5)

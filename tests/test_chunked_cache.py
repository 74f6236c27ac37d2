"""Cache groups whose layers see chunks of positions: which pages a request holds, what comes back
when a chunk ends, and what later requests may share.  No GPU."""
from __future__ import annotations

import pytest
import torch

from helix_runtime_b200.cache.manager import CacheManager, KvNeed


def manager(need, pages=12, page_size=8, slack=0, window_pages=None, poison=False):
    return CacheManager({0: need}, {}, page_size, pages, 2, 1024, torch.float32,
                        torch.device("cpu"), poison=poison, window_slack_pages=slack,
                        window_pages=window_pages)


def live_pages(cache, request):
    return [index for index, page in enumerate(cache._requests[request].tables[0]) if page >= 0]


def test_what_a_position_sees():
    need = KvNeed(1, 8, chunk=10)
    assert [need.first_seen(p) for p in (0, 9, 10, 19, 20, 35)] == [0, 0, 10, 10, 20, 30]
    assert need.reach == 10 and need.bounded
    both = KvNeed(1, 8, window=4, chunk=10)
    assert [both.first_seen(p) for p in (0, 3, 4, 9, 10, 12, 15)] == [0, 0, 1, 6, 10, 10, 12]
    assert both.reach == 4
    assert KvNeed(1, 8).first_seen(77) == 0 and KvNeed(1, 8).reach is None
    with pytest.raises(ValueError):
        KvNeed(1, 8, chunk=10, keep_first=2)


@pytest.mark.parametrize("chunk", [1, 5, 8, 13, 16, 40])
@pytest.mark.parametrize("sizes", [(1,) * 100, (7, 2, 30, 3, 41, 1, 1, 15)])
def test_pages_come_back_when_their_chunk_has_ended(chunk, sizes):
    cache = manager(KvNeed(1, 8, chunk=chunk), pages=16)
    cache.admit("a")
    length = 0
    for size in sizes:
        cache.extend("a", length + size)
        length += size
        cache.commit("a", length)
        first = length // chunk * chunk // 8      # of the next position's chunk
        assert live_pages(cache, "a") == list(range(first, -(-length // 8)))
        cache.check()
    cache.release("a")
    cache.check()
    assert cache.free_pages() == [16]


def test_a_pool_of_the_size_that_is_promised_serves_any_length():
    need = KvNeed(1, 8, chunk=20)
    for slack in (0, 1):
        cache = manager(need, pages=64, slack=slack)
        pages = cache.pages_needed_alone(500)[0]
        small = manager(need, pages=pages, slack=slack)
        small.admit("a")
        for length in range(1, 501):
            small.extend("a", length)
            small.commit("a", length)
        small.check()


def test_chunked_groups_may_have_a_pool_of_their_own():
    cache = CacheManager({0: KvNeed(1, 8), 1: KvNeed(1, 8, chunk=20)}, {}, 8, 30, 2, 1024,
                         torch.float32, torch.device("cpu"), window_pages={20: 7})
    assert sorted(cache.free_pages()) == [7, 30]
    assert cache.shares_whole_prefixes_only
    with pytest.raises(ValueError):
        manager(KvNeed(1, 8, chunk=20), window_pages={21: 7})


def test_a_prefix_is_held_and_adopted_across_a_chunks_end():
    """A prompt of 43 tokens in chunks of 20: its last page boundary, 40, is a chunk's end, so the
    prefix holds no page and a request that adopts it needs none; at 42 tokens with pages of 6
    the prefix's last chunk has begun and its pages are shared."""
    cache = manager(KvNeed(1, 8, chunk=20), slack=1)
    cache.admit("a")
    cache.extend("a", 43)
    cache.commit("a", 43)
    assert cache.hold("p", "a", 40) == 0
    assert cache.adopt("b", "p") is not None
    assert cache.length("b") == 40 and live_pages(cache, "b") == []
    cache.check()
    for request in ("a", "b"):
        cache.release(request)
    cache.drop("p")
    cache.check()
    cache = manager(KvNeed(1, 8, chunk=20), page_size=6, slack=1)
    cache.admit("a")
    cache.extend("a", 45)
    cache.commit("a", 45)
    assert cache.hold("p", "a", 42) == 1                      # page 6: positions 36 to 41
    cache.adopt("b", "p")
    assert live_pages(cache, "b") == [6]
    cache.check()


def test_with_slack_the_pages_in_front_of_a_chunks_end_stay_until_a_page_later():
    """The prefix that is published ends at a page boundary up to a page short of its request: a
    chunk that ended in between is still there."""
    cache = manager(KvNeed(1, 8, chunk=20), slack=1)
    cache.admit("a")
    cache.extend("a", 41)
    cache.commit("a", 39)
    assert live_pages(cache, "a") == [2, 3, 4, 5]
    cache.commit("a", 41)
    assert live_pages(cache, "a") == [2, 3, 4, 5]             # 41 - 8 lies in the chunk of 20
    assert cache.hold("p", "a", 32) == 2
    cache.extend("a", 48)
    cache.commit("a", 48)
    assert live_pages(cache, "a") == [5]
    cache.check()

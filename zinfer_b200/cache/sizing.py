"""How many pages a byte budget buys, and what a pool costs.

One page of a group holds ``page_size`` tokens of keys and of values for every
cache of the group: ``caches * 2 * kv heads * page_size * head_dim * element size``
bytes (half of that in a group that keeps keys only; with values of another size than the keys, key size plus
value size in place of twice the head size).  Every group gets the same number of pages, so one page id across all groups
costs the sum of those; only a group whose entries stand for P tokens each gets a P-th of them, and one page per request
beside, since every request may have begun a page of it.  The reference sizes one contiguous cache per request by
the same product over its layers
(src/model/runtime/optimized_kv_cache/cache.zig:423-456) and prints it with its
benchmarks (src/app/cli/tools/bench/runtime.zig:74-79).
"""
from __future__ import annotations

from typing import Optional


def entry_pages(num_pages: int, tokens_per_entry: int, requests: int) -> int:
    """Pages of a group beside groups of ``num_pages`` pages of tokens, when its entries stand for several tokens."""
    return num_pages if tokens_per_entry <= 1 else -(-num_pages // tokens_per_entry) + requests


def group_shapes(kv_needs: dict) -> list[tuple[int, int, int, int]]:
    """(caches, kv heads, elements per entry and kv head, tokens per entry) per group, grouping equal needs like the manager
    does; the elements are key size plus value size (the key size alone in a group that keeps keys only)."""
    groups: dict[tuple, int] = {}
    for need in kv_needs.values():
        values = getattr(need, "values", True)
        vd = getattr(need, "value_dim", None) or need.head_dim
        keep = (getattr(need, "keep_first", 0) or 0) if need.window is not None else 0
        per = int(getattr(need, "tokens_per_entry", 1) or 1)
        key = (need.num_kv_heads, need.head_dim, need.window, values, vd if values else 0, keep, per)
        groups[key] = groups.get(key, 0) + 1
    return [(n, key[0], key[1] + key[4], key[6]) for key, n in groups.items()]


def bytes_per_page(kv_needs: dict, page_size: int, element_size: int) -> int:
    """Bytes that one more page of tokens costs across all groups (a P-th of a page where an entry stands for P tokens)."""
    return sum(-(-n * heads * page_size * d * element_size // per) for n, heads, d, per in group_shapes(kv_needs))


def bytes_per_token(kv_needs: dict, element_size: int) -> int:
    return bytes_per_page(kv_needs, 1, element_size)


def pages_for(kv_needs: dict, page_size: int, element_size: int, *, budget_bytes: Optional[int] = None,
              tokens: Optional[int] = None, requests: int = 0) -> int:
    """Pages per group: what ``budget_bytes`` buys (floor), at most what ``tokens`` need
    (each rounded up to whole pages); at least one.  ``requests``: how many requests may be live, for the pages that
    groups with several tokens per entry hold beside (:func:`entry_pages`)."""
    per_page = bytes_per_page(kv_needs, page_size, element_size)
    if budget_bytes is not None:
        budget_bytes -= sum(n * heads * page_size * d * element_size * (requests + 1)
                            for n, heads, d, per in group_shapes(kv_needs) if per > 1)
    pages = None
    if budget_bytes is not None and per_page > 0:
        pages = max(0, budget_bytes) // per_page
    if tokens is not None:
        want = -(-tokens // page_size)
        pages = want if pages is None else min(pages, want)
    if pages is None:
        raise ValueError("give a byte budget or a token count")
    return max(1, int(pages))

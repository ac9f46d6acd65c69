"""What the cache manager has to know about a kind of per-request state, registered per `StateNeed` class.

The reference's planner reads only a layer's `StateNeed` (crates/kf-core/src/layer.rs:29-43: `KvCache`, `Recurrent`,
`TokenShift`, `Latent`, ...) and never the layer type; each variant brings its own row width and lifetime.  Here a
state kind is an object with the few answers the manager and the sizing need, and a new kind is registered from
wherever its mixer is defined (a test file is enough): the manager has no list of kinds of its own.

A *paged* kind stores something for every token, in pages that the manager hands out; its answers:
  window(need)                          -> tokens that stay readable (None: all); needs with equal windows share a
                                           group, i.e. a pool of page ids and one block table per request
  chunk(need)       (optional)          -> instead of a window: the size of the runs of positions, counted from a request's
                                           start, outside of which nothing is read (None)
  keep_first(need)  (optional)          -> tokens at the start of a request that stay readable behind the window (0);
                                           needs of one group agree on it too
  page_shape(need, page_size)           -> shape of one page of one cache slot
  page_bytes(need, page_size, elsize)   -> its bytes (elsize: bytes of the cache's element type)
  dtype(need, cache_dtype)              -> element type of the storage
  view(storage, page_size, group, writes, need) -> what the mixer's forward() is given
A *fixed* kind stores one state of fixed shape per live request, zeroed at admission:
  shape(need), dtype(need, cache_dtype), fixed_bytes(need), view(storage, writes, need)
"""
from __future__ import annotations

import math

import torch

from ..parts.base import FixedState, PagedKV, StateBundle


class PagedKVView:
    """What a mixer sees of a cache slot of keys and values during one step."""

    def __init__(self, pages: torch.Tensor, page_size: int, group: int, writes: bool):
        self.pages = pages              # [n_pages, 2 (key, value), n_kv_heads, page_size, head_dim]
        self.page_size = page_size
        self.group = group
        self.writes = writes


class FixedStateView:
    def __init__(self, state: torch.Tensor, writes: bool):
        self.state = state              # [max_requests, *shape]; row = the request's state slot
        self.writes = writes


class PagedKVKind:
    paged = True

    def window(self, need):
        return need.window

    def chunk(self, need):
        return getattr(need, "chunk", None)

    def keep_first(self, need):
        return int(getattr(need, "keep_first", 0) or 0) if need.window is not None else 0

    def page_shape(self, need, page_size):
        return (2, need.n_kv_heads, page_size, need.head_dim)

    def page_bytes(self, need, page_size, elsize):
        return 2 * need.n_kv_heads * page_size * need.head_dim * elsize

    def dtype(self, need, cache_dtype):
        return cache_dtype

    def view(self, storage, page_size, group, writes, need):
        return PagedKVView(storage, page_size, group, writes)


class FixedStateKind:
    paged = False

    def shape(self, need):
        return tuple(need.shape)

    def dtype(self, need, cache_dtype):
        return need.dtype

    def fixed_bytes(self, need):
        return int(math.prod(need.shape)) * torch.empty(0, dtype=need.dtype).element_size()

    def view(self, storage, writes, need):
        return FixedStateView(storage, writes)


def lifetime_of(need, kind):
    """What names a paged need's group: its window alone, (window, kept first tokens) when some are kept, or
    ("chunk", size).  The reach in tokens, the kept tokens and whether it is chunks are `lifetime_window`,
    `lifetime_keep` and `lifetime_chunked` of that key."""
    chunk = kind.chunk(need) if hasattr(kind, "chunk") else None
    if chunk is not None:
        return ("chunk", int(chunk))
    window = kind.window(need)
    keep = int(kind.keep_first(need)) if (window is not None and hasattr(kind, "keep_first")) else 0
    return (window, keep) if keep > 0 else window


def lifetime_chunked(key) -> bool:
    return isinstance(key, tuple) and key[0] == "chunk"


def lifetime_window(key):
    if lifetime_chunked(key):
        return key[1]
    return key[0] if isinstance(key, tuple) else key


def lifetime_keep(key) -> int:
    return key[1] if isinstance(key, tuple) and not lifetime_chunked(key) else 0


def lifetime_name(key) -> str:
    """The key in words, without spaces: none, 96, 96+4 (four kept tokens), chunk200."""
    if lifetime_chunked(key):
        return f"chunk{key[1]}"
    return "none" if key is None else (f"{key[0]}+{key[1]}" if isinstance(key, tuple) else str(key))


def flatten_need(need) -> list:
    """The plain needs behind one cache slot: a bundle's parts in order, a single need as a list of one, none as []."""
    if need is None:
        return []
    if isinstance(need, StateBundle):
        out = []
        for part in need.parts:
            out += flatten_need(part)
        return out
    return [need]


_KINDS: dict = {}


def register_state_kind(need_class: type, kind) -> None:
    """Make the manager able to hold what `need_class` declares.  `kind` answers the questions in this module's
    header (see `PagedKVKind` and `FixedStateKind`)."""
    if need_class in _KINDS and type(_KINDS[need_class]) is not type(kind):
        raise ValueError(f"a state kind for {need_class.__name__} is already registered")
    _KINDS[need_class] = kind


def kind_of(need):
    for cls in type(need).__mro__:
        if cls in _KINDS:
            return _KINDS[cls]
    raise TypeError(f"unknown state need {need!r}: no state kind is registered for {type(need).__name__} "
                    f"(known: {sorted(c.__name__ for c in _KINDS)})")


register_state_kind(PagedKV, PagedKVKind())
register_state_kind(FixedState, FixedStateKind())

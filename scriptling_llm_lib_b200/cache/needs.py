"""What a mixer asks of the cache for its layer."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

PAGE = 64  # tokens per page; the kernel libraries are compiled with the same number and say so when loaded

# kind of cache -> first position that a query at position >= length can still see (pages wholly
# below it are given back to the pool at once). "full" keeps everything; "window" the last
# `window` positions. A mixer with another retention rule registers its kind here.
CACHE_KINDS: dict[str, Callable[["CacheNeed", int], int]] = {}


def register_cache_kind(kind: str, first_needed: Callable[["CacheNeed", int], int], replace: bool = False) -> None:
    if kind in CACHE_KINDS and not replace:
        raise ValueError(f"cache kind {kind!r} is already registered")
    CACHE_KINDS[kind] = first_needed


@dataclass(frozen=True)
class CacheNeed:
    """Keys and values per position: `kind` says which positions must be kept ("full": all;
    "window": the last `window`; "chunk": the chunk of `window` positions the next query lies in; or a registered kind
    of the mixer's own). `keep`: a sequence's first positions that are kept whatever the kind gives back."""
    kind: str
    kv_heads: int
    head_dim: int
    window: int | None = None
    v_dim: int | None = None      # width of a value head where it differs from the keys' (None: head_dim)
    keep: int = 0

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_dim is None else self.v_dim

    def __post_init__(self):
        if self.kind not in CACHE_KINDS:
            raise ValueError(f"cache kind {self.kind!r}; known: {', '.join(sorted(CACHE_KINDS))}")
        if (self.kind in ("window", "chunk")) != (self.window is not None) and self.kind in ("full", "window", "chunk"):
            raise ValueError("a window or chunk cache needs its size, a full cache has none")
        if self.keep < 0:
            raise ValueError(f"a cache that keeps the first {self.keep} positions")

    def first_needed(self, length: int) -> int:
        return CACHE_KINDS[self.kind](self, length)

    def pages_seen(self) -> int | None:
        """The most pages one query can see (None: no bound but its sequence)."""
        if self.window is None or self.kind not in ("window", "chunk"):
            return None
        return (self.window + 2 * PAGE - 2) // PAGE + (self.keep + PAGE - 1) // PAGE


register_cache_kind("full", lambda need, length: 0)
register_cache_kind("window", lambda need, length: length - need.window + 1)
# chunks of `window` positions counted from 0: a later query sees nothing before the start of the chunk `length` lies in
register_cache_kind("chunk", lambda need, length: length - length % need.window)


@dataclass(frozen=True)
class StateNeed:
    """Per-sequence state of fixed size (a recurrent mixer's carry): zeroed when a slot is opened.
    A part with several such tensors (a recurrence's carry and the last inputs of its short
    convolutions) answers `state_need()` with a dict name -> StateNeed; the unit's state is then a
    dict of tensors under the same names."""
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32

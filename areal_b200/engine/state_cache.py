"""Memory of running requests: the page pool every cache is built on, and the cache of mixer stacks (pages of keys and
values, or of latents, per attention layer, one state slot per request for the recurrent layers)."""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional

import torch


class PagePool:
    """Free list and reference counts of fixed-size pages."""

    def __init__(self, num_pages: int, page_size: int):
        self.page_size, self.num_pages = page_size, num_pages
        self.reset_pages()

    def reset_pages(self) -> None:
        self.free = list(range(self.num_pages - 1, -1, -1))
        self.ref = [0] * self.num_pages     # users of a page: its sequence, plus the prefix cache and other sequences when shared

    def alloc(self, n: int) -> Optional[list[int]]:
        if len(self.free) < n:
            return None
        out = self.free[-n:] if n else []
        if n:
            del self.free[-n:]
        for p in out:
            self.ref[p] = 1
        return out

    def share(self, pages: list[int]) -> None:
        for p in pages:
            self.ref[p] += 1

    def release(self, pages: list[int]) -> None:
        for p in pages:
            self.ref[p] -= 1
            if self.ref[p] <= 0:
                self.ref[p] = 0
                self.free.append(p)

    def pages_needed(self, tokens: int) -> int:
        return (tokens + self.page_size - 1) // self.page_size


@dataclass
class Carried:
    """What one request holds between steps: its state slot and the pages from number ``first_page`` of its sequence on
    (pages that no layer can see any more have been given back)."""

    slot: int
    pages: list[int] = field(default_factory=list)
    first_page: int = 0
    length: int = 0              # tokens absorbed


SLOT_STATES = ("tail", "state", "shift")       # what a layer may keep per request


class LayerCache:
    __slots__ = ("k", "v", "key_factor") + SLOT_STATES

    def __init__(self):
        for name in self.__slots__:
            setattr(self, name, None)


class StateCache(PagePool):
    """Pages for the attention layers (``[pages * page_size, heads, dim]`` of K and V per layer, each with its own sizes; a
    layer whose keys and values come from one latent, or whose keys are its values, has K only, and a number per key beside it
    when keys are normed as they are read) and fp32 slots for what else a layer carries (convolution tails, recurrence states,
    the row before for a token shift). A slot is not cleared when it changes hands: kernels take the state of a request that has absorbed
    nothing as zero."""

    def __init__(self, mixers: list, num_pages: int, page_size: int, num_slots: int, device, dtype):
        super().__init__(num_pages, page_size)
        self.num_slots = num_slots
        self.layers: list[LayerCache] = []
        self._sight: dict = {}       # attention layers that see the same stretch of positions, once each
        self.windows: set = set()    # sliding windows of the latent layers
        for mx in mixers:
            lc, shapes = LayerCache(), mx.memory()
            if "kv" in shapes:
                lc.k, lc.v = (None if s is None else torch.zeros(num_pages * page_size, *s, device=device, dtype=dtype) for s in shapes["kv"])
                if "key_factor" in shapes:
                    lc.key_factor = torch.zeros(num_pages * page_size, *shapes["key_factor"], device=device, dtype=torch.float32)
                self._sight[type(mx), mx.span] = mx
                if mx.lists_pages:
                    self.windows.add(mx.span)
            for name in SLOT_STATES:
                if name in shapes:
                    setattr(lc, name, torch.zeros(num_slots, *shapes[name], device=device, dtype=torch.float32))
            self.layers.append(lc)
        self.has_kv = bool(self._sight)
        spans = [mx.span for mx in self._sight.values()]
        # positions the furthest-seeing layer may look at (0: all of them)
        self.span = 0 if not spans or min(spans) == 0 else max(spans)
        self.free_slots = list(range(num_slots - 1, -1, -1))

    @staticmethod
    def bytes_per_page(mixers: list, page_size: int, elem: int) -> int:
        n = 0
        for mx in mixers:
            shapes = mx.memory()
            n += sum(s[0] * s[1] for s in shapes.get("kv", ()) if s) * elem + sum(shapes.get("key_factor", ())) * 4
        return n * page_size

    @staticmethod
    def bytes_per_slot(mixers: list) -> int:
        return sum(4 * math.prod(s) for mx in mixers for name, s in mx.memory().items() if name in SLOT_STATES)

    def first_visible(self, pos: int) -> int:
        """Earliest position that a query at ``pos`` or later can see in any attention layer."""
        return 0 if self.span == 0 else min(mx.first_visible(pos) for mx in self._sight.values())

    def table_width(self, context: int) -> int:
        """Page-table columns a single-token step needs at most."""
        full = context // self.page_size + 1
        return full if self.span == 0 else min(full, self.span // self.page_size + 2)

    def open(self) -> Optional[Carried]:
        return Carried(self.free_slots.pop()) if self.free_slots else None

    def pages_to_grow(self, c: Carried, total: int) -> int:
        if not self.has_kv:
            return 0
        return max(0, self.pages_needed(total) - c.first_page - len(c.pages))

    def grow(self, c: Carried, total: int) -> bool:
        """Pages for ``total`` tokens of the sequence; False (nothing taken) when the pool is short."""
        got = self.alloc(self.pages_to_grow(c, total))
        if got is None:
            return False
        c.pages += got
        return True

    def advance(self, c: Carried, n: int) -> None:
        """``n`` more tokens were absorbed; gives back the pages that fell out of every layer's sight."""
        c.length += n
        drop = min(self.first_visible(c.length) // self.page_size - c.first_page, len(c.pages))
        if drop > 0:
            self.release(c.pages[:drop])
            del c.pages[:drop]
            c.first_page += drop

    def close(self, c: Carried) -> None:
        self.release(c.pages)
        c.pages = []
        self.free_slots.append(c.slot)
        c.slot = -1

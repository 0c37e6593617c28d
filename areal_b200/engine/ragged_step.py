"""One step of a mixer stack over a ragged batch: several requests, each bringing any number of its next tokens
(a whole prompt, a portion of one, or the token it has just sampled), from the pages and state slots that earlier steps
left. The rollout engine's generation loop and the trace runner both step through :class:`RaggedRunner`.

Requests with one new token come first in the batch, so that they take the decode kernels; a step of single tokens only
runs as a CUDA graph over static buffers (one host-to-device copy per step)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import numpy as np
import torch

from ..ops import lib as oplib
from ..ops.mixer_ops import ATTN_TILE, SCAN_BLOCK, PageList, RaggedBatch
from .state_cache import Carried, StateCache

DECODE_BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 256, 512)


@dataclass
class Entry:
    carry: Carried
    tokens: list
    want: list           # places among ``tokens`` whose logits are asked for


class RaggedRunner:
    def __init__(self, model, cache: StateCache, device, max_batch: int, context_length: int, use_graph: bool = True):
        self.model, self.cache, self.device = model, cache, torch.device(device)
        self.max_batch = max_batch
        self.width = max(1, cache.table_width(context_length))
        # positions that have a learned vector (None: positions are not limited)
        self.max_positions = model.cfg.max_position_embeddings if model.cfg.learned_positions else None
        # the routing kernel takes up to 256 experts, 16 per token; beyond that the choice reads back to the host
        moe = [m["mlp"]["router"] for m in model.cfg.mixer_layers if m["mlp"] and m["mlp"]["kind"] == "moe"]
        self.use_graph = use_graph and self.device.type == "cuda" and all(r["experts"] <= 256 and r["top"] <= 16 for r in moe)
        self._graphs: dict = {}
        self._static: dict = {}
        self.stream: Optional[torch.cuda.Stream] = None      # set by the engine: graphs are captured on the stream that replays them

    # ------------------------------------------------------------------ batch layout
    def _upload(self, pieces: list) -> list:
        """One copy for all index arrays of a step; every piece starts on a 16-byte boundary."""
        offs, n = [], 0
        for a in pieces:
            offs.append(n)
            n += -(-a.size // 4) * 4
        flat = torch.zeros(n, dtype=torch.int32, pin_memory=self.device.type == "cuda")
        host = flat.numpy()
        for a, o in zip(pieces, offs):
            host[o:o + a.size] = a.reshape(-1)
        dev = flat.to(self.device, non_blocking=True)
        return [dev[o:o + a.size].view(a.shape) for a, o in zip(pieces, offs)]

    def _page_rows(self, entries: list, width: int) -> np.ndarray:
        pt = np.zeros((len(entries), width), np.int32)
        for i, e in enumerate(entries):
            pt[i, :len(e.carry.pages)] = e.carry.pages
        return pt

    def _layout(self, entries: list):
        ps = self.cache.page_size
        n = np.array([len(e.tokens) for e in entries], np.int64)
        start = np.array([e.carry.length for e in entries], np.int64)
        cu = np.concatenate([[0], np.cumsum(n)])
        row_entry = np.repeat(np.arange(len(entries)), n)
        pos = np.arange(cu[-1]) - cu[row_entry] + start[row_entry]
        base = np.array([e.carry.first_page for e in entries], np.int64)
        pt = self._page_rows(entries, max([1] + [len(e.carry.pages) for e in entries]))
        slots = pt[row_entry, pos // ps - base[row_entry]].astype(np.int64) * ps + pos % ps if self.cache.has_kv else pos * 0
        n_dec = int((n == 1).sum())
        blocks, tiles = [], []
        sight = getattr(self.cache, "first_visible", lambda p: 0)
        for i in range(n_dec, len(entries)):
            for r in range(0, int(n[i]), SCAN_BLOCK):
                blocks.append((i, cu[i] + r, min(SCAN_BLOCK, n[i] - r), int(r == 0)))
            tiles += [(i, cu[i] + r) for r in range(0, int(n[i]), ATTN_TILE)]
        # tiles that see the most keys start first: the last ones to run are short
        tiles.sort(key=lambda t: sight(int(pos[t[1]])) - pos[t[1]])
        toks = np.concatenate([np.asarray(e.tokens, np.int64) for e in entries])
        state = np.array([e.carry.slot for e in entries])
        arrs = [toks, pos, slots, row_entry, cu, start, state, pt, base]
        if blocks:
            arrs += [np.array(blocks), np.array(tiles)]
        windows = sorted(getattr(self.cache, "windows", ())) if blocks else []
        for w in windows:
            arrs += self._visible_pages(entries, n_dec, start, n, base, w)
        want = [cu[i] + w for i, e in enumerate(entries) for w in e.want]
        arrs.append(np.array(want, np.int64))
        up = self._upload([a.astype(np.int32) for a in arrs])
        seen = {w: PageList(*up[11 + 3 * i:14 + 3 * i]) for i, w in enumerate(windows)}
        b = RaggedBatch(*up[:9], blocks=up[9] if blocks else None, tiles=up[10] if blocks else None, n_dec=n_dec, page_size=ps, seen=seen)
        return b, up[-1]

    def _visible_pages(self, entries: list, n_dec: int, start, n, base, window: int) -> list:
        """Pages that the portions of a step see through a sliding window, one after the other; and, per entry, the table
        of their numbers in that list with the page of the sequence that it begins with."""
        ps = self.cache.page_size
        first = np.maximum(start - window + 1, 0) // ps if window else start * 0
        last = (start + n - 1) // ps
        count = np.where(np.arange(len(entries)) >= n_dec, last - first + 1, 0)
        table, pages = np.zeros((len(entries), max(1, count.max())), np.int64), []
        for i in range(n_dec, len(entries)):
            table[i, :count[i]] = len(pages) + np.arange(count[i])
            pages += entries[i].carry.pages[first[i] - base[i]:last[i] - base[i] + 1]
        return [np.array(pages), table, first]

    # ------------------------------------------------------------------ the step
    @torch.no_grad()
    def step(self, entries: list, on_layer=None) -> Optional[torch.Tensor]:
        """Absorbs every entry's tokens. Returns the fp32 logits of the wanted places ``[n, vocab]``, in the order of
        the entries and of their ``want`` (None when nothing is wanted). The caller has grown the pages."""
        for e in entries:
            held = (e.carry.first_page + len(e.carry.pages)) * self.cache.page_size
            if not e.tokens or (self.cache.has_kv and held < e.carry.length + len(e.tokens)):
                raise ValueError("an entry of a step needs tokens, and pages for all of them")
            if self.max_positions is not None and e.carry.length + len(e.tokens) > self.max_positions:
                raise ValueError(f"a sequence of this model has at most {self.max_positions} tokens")
        if self.use_graph and on_layer is None and len(entries) <= self.max_batch and all(
                len(e.tokens) == 1 and e.want == [0] and len(e.carry.pages) <= self.width for e in entries):
            out = self._decode_graph(entries)
        else:
            out = self._run(entries, on_layer)
        for e in entries:
            self.cache.advance(e.carry, len(e.tokens))
        return out

    def _run(self, entries: list, on_layer):
        order = sorted(range(len(entries)), key=lambda i: len(entries[i].tokens) != 1)
        ent = [entries[i] for i in order]
        b, want = self._layout(ent)
        hidden = self.model.forward_step(b, self.cache, on_layer)
        if want.numel() == 0:
            return None
        logits = self.model.logits(hidden.index_select(0, want))
        if order != sorted(order):
            # back to the caller's order of entries
            first, n = {}, 0
            for i in order:
                first[i] = n
                n += len(entries[i].want)
            idx = [first[i] + w for i in range(len(entries)) for w in range(len(entries[i].want))]
            logits = logits.index_select(0, torch.tensor(idx, device=logits.device))
        return logits

    # ------------------------------------------------------------------ single tokens: CUDA graph over static buffers
    def _bucket(self, n: int) -> int:
        return next(b for b in DECODE_BUCKETS if b >= n)

    def _static_of(self, B: int):
        st = self._static.get(B)
        if st is None:
            cols = 6 + self.width
            host = torch.zeros(B * cols, dtype=torch.int32).pin_memory()
            dev = torch.zeros(B * cols, dtype=torch.int32, device=self.device)
            part = lambda t, i: t[i * B:(i + 1) * B]      # noqa: E731
            ar = torch.arange(B + 1, dtype=torch.int32, device=self.device)
            b = RaggedBatch(tokens=part(dev, 0), pos=part(dev, 1), slots=part(dev, 2), row_entry=ar[:B], cu=ar, start=part(dev, 3),
                            state=part(dev, 4), page_base=part(dev, 5), pages=dev[6 * B:].view(B, self.width), blocks=None, tiles=None,
                            n_dec=B, page_size=self.cache.page_size)
            st = self._static[B] = (host, host.numpy().reshape(-1), dev, b, torch.cuda.Event())
        return st

    def _decode_graph(self, entries: list) -> torch.Tensor:
        n, ps = len(entries), self.cache.page_size
        B = self._bucket(n)
        host, h, dev, b, copied = self._static_of(B)
        copied.synchronize()                 # the previous step's copy has read the pinned buffer
        part = lambda i: h[i * B:(i + 1) * B]             # noqa: E731
        length = np.array([e.carry.length for e in entries], np.int32)
        base = np.array([e.carry.first_page for e in entries], np.int32)
        pt = self._page_rows(entries, self.width)
        for i in range(6):
            part(i)[n:] = -1 if i in (2, 4) else 0        # padding rows: no cache row, no slot
        part(0)[:n] = [e.tokens[0] for e in entries]
        part(1)[:n] = part(3)[:n] = length
        part(2)[:n] = pt[np.arange(n), length // ps - base] * ps + length % ps if self.cache.has_kv else 0
        part(4)[:n] = [e.carry.slot for e in entries]
        part(5)[:n] = base
        h[6 * B:].reshape(B, self.width)[:n] = pt
        g = self._graphs.get(B)
        if g is None:
            g = self._capture(B, b, dev)
        dev.copy_(host, non_blocking=True)
        copied.record()
        graph, logits, kernels = g
        graph.replay()
        oplib.LAUNCHES["count"] += kernels
        return logits[:n]

    def _capture(self, B: int, b: RaggedBatch, dev: torch.Tensor):
        def forward():
            return self.model.logits(self.model.forward_step(b, self.cache))

        # warm-up and capture run on padding rows only: they leave the cache and every state slot alone
        dev.zero_()
        b.slots.fill_(-1)
        b.state.fill_(-1)
        for _ in range(2):
            forward()
        torch.cuda.current_stream().synchronize()
        graph = torch.cuda.CUDAGraph()
        n0 = oplib.launch_count()
        with torch.cuda.graph(graph, stream=self.stream, capture_error_mode="thread_local"):
            logits = forward()
        kernels = oplib.launch_count() - n0
        oplib.LAUNCHES["count"] = n0
        self._graphs[B] = (graph, logits, kernels)
        return self._graphs[B]

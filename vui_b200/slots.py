"""Slots, buckets, graphs and batching shared by the engines.

An engine owns a cache of ``max_rows + 1`` slots of ``max_seq`` positions (the spare slot is what padded rows of a
graph aim at), hands slots out as rows, packs the prefills of several rows into calls of at most ``max_prefill_rows``,
captures one CUDA graph per batch-size bucket, and refills finished slots from a queue.  ``Engine`` (speech) and
``TokenEngine`` (token models) are this plus what a step of their model is.
"""

from __future__ import annotations

import ctypes as C
from collections import deque

import torch

from . import _lib


def _make_buckets(max_bs: int) -> list[int]:
    out, b = [], 1
    while b < max_bs:
        out.append(b)
        b *= 2
    if not out or out[-1] != max_bs:
        out.append(max_bs)
    return out


def _get_bucket(n: int, buckets: list[int]) -> int:
    for b in buckets:
        if n <= b:
            return b
    return buckets[-1]


def _ptr(t):
    return C.c_void_p(t.data_ptr()) if t is not None else None


class SlotEngine:
    """Base of the engines.  A subclass sets ``_ABI`` (the prefix of its library's functions) and ``_ROW`` (its row
    class), and provides ``device``, ``_lib``, ``_handle`` and ``seq_lens`` before rows are taken."""

    _ABI = "vuib_"
    _ROW: type

    def _init_slots(self, max_rows: int) -> None:
        self.max_rows = max_rows
        self._pad_slot = max_rows
        self._buckets = _make_buckets(max_rows)
        self._free: set[int] = set(range(max_rows))
        self._rows: dict = {}

    def _fn(self, name: str):
        return getattr(self._lib, self._ABI + name)

    def _ck(self, code: int) -> None:
        _lib.check(self._handle, code, self._fn("last_error"))

    @property
    def _stream(self):
        return C.c_void_p(torch.cuda.current_stream(self.device).cuda_stream)

    def __del__(self):
        try:
            if self._handle:
                self._fn("destroy")(self._handle)
                self._handle = C.c_void_p()
        except Exception:
            pass

    def launch_count(self) -> int:
        return int(self._fn("launch_count")(self._handle))

    def check_device(self) -> None:
        """Raise if a kernel saw a slot, position or code out of range."""
        self._ck(self._fn("check_device_flag")(self._handle, self._stream))

    # ---------------------------------------------------------- row lifecycle
    def new_row(self):
        if not self._free:
            raise RuntimeError(f"No free rows (max_rows={self.max_rows} all in use)")
        idx = min(self._free)
        self._free.remove(idx)
        row = self._ROW(self, idx)
        self._rows[idx] = row
        self._set_len(idx, 0)
        return row

    def _release_row(self, row) -> None:
        self._rows.pop(row.idx, None)
        self._free.add(row.idx)

    def reset(self) -> None:
        for row in list(self._rows.values()):
            row.close()
        self.seq_lens.zero_()

    def _set_len(self, slot: int, n: int) -> None:
        self.seq_lens[slot] = n

    def _rewind_row(self, row, offset: int) -> int:
        self._set_len(row.idx, offset)
        return offset

    # ---------------------------------------------------------------- prefill
    def _pack_rows(self, items, run) -> None:
        """Cut (row, tensor of n positions) items into calls of at most ``max_prefill_rows`` positions:
        ``run(list of (slot, first position, piece, item index))`` per call.  An item longer than one call is cut; a
        slot may appear several times in a call (its pieces carry consecutive positions, and every piece is in the
        cache before any attends)."""
        pend: list[tuple] = []
        offsets: dict[int, int] = {}
        used = 0
        for k, (row, t) in enumerate(items):
            n_all = t.shape[0]
            off = offsets[row.idx] if row.idx in offsets else row.offset
            if off + n_all > self.max_seq:
                raise RuntimeError(f"prefill of {n_all} positions overflows max_seq={self.max_seq}")
            start = 0
            while start < n_all:
                if used == self.max_prefill_rows:
                    run(pend)
                    pend, used = [], 0
                n = min(self.max_prefill_rows - used, n_all - start)
                pend.append((row.idx, off + start, t[start:start + n], k))
                used += n
                start += n
            offsets[row.idx] = off + n_all
        if pend:
            run(pend)

    # ----------------------------------------------------------------- graphs
    def _capture_graph(self, call, keep) -> torch.cuda.CUDAGraph:
        """Capture ``call()`` after one run of it on a side stream (which loads the kernels) with every row aimed at
        the spare slot and lengths frozen; the tensors of ``keep`` are put back afterwards."""
        saved = [t.clone() for t in (self._g_slot_idx, self._g_seq_inc, self.seq_lens, *keep)]
        self._g_slot_idx.fill_(self._pad_slot)
        self._g_seq_inc.zero_()
        self.seq_lens[self._pad_slot] = 0
        torch.cuda.synchronize(self.device)
        side = torch.cuda.Stream(self.device)
        side.wait_stream(torch.cuda.current_stream(self.device))
        with torch.cuda.stream(side):
            call()
        torch.cuda.current_stream(self.device).wait_stream(side)
        torch.cuda.synchronize(self.device)
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            call()
        torch.cuda.synchronize(self.device)
        for t, old in zip((self._g_slot_idx, self._g_seq_inc, self.seq_lens, *keep), saved):
            t.copy_(old)
        return g

    def _pad_to_bucket(self, n: int) -> int:
        """The bucket of n active rows; the static rows above n are aimed at the spare slot."""
        B = _get_bucket(n, self._buckets)
        if n < B:
            self._g_slot_idx[n:B].fill_(self._pad_slot)
            self._g_seq_inc[n:B].zero_()
        return B

    # ---------------------------------------------------- continuous batching
    def _run_continuous(self, n_requests: int, admit, step) -> None:
        """More requests than slots: ``admit(list of (request, slot))`` starts requests and returns {slot: state} of
        those that go on; ``step(slots, states)`` advances all of them and returns the slots that are finished, which
        are refilled from the queue."""
        pending: deque[int] = deque(range(n_requests))
        free = set(range(self.max_rows))
        active: dict = {}

        def backfill() -> None:
            while pending and free:
                batch = []
                while pending and free:
                    slot = min(free)
                    free.remove(slot)
                    batch.append((pending.popleft(), slot))
                started = admit(batch)
                for _, slot in batch:
                    if slot in started:
                        active[slot] = started[slot]
                    else:
                        self._rows.pop(slot, None)
                        free.add(slot)

        backfill()
        while active:
            slots = sorted(active)
            for s in step(slots, [active[s] for s in slots]):
                active.pop(s)
                self._rows.pop(s, None)
                free.add(s)
            backfill()

"""Recurrent state of requests, for layers that carry one instead of (or besides) a KV cache.

One fp32 row per request slot (the request table's row numbers, the hold row of padded decode batches included) holds the
state of all layers back to back, so that a snapshot is one row copy.  A layer asks for its room with `reserve` and gets
its view with `view`: [rows, elements], row pitch `row_elems`.  Kernels start from zero when a request's first token is at
position 0, so a slot needs no clearing when it is used again.

`RecurrentStateMixin` gives a model the snapshot interface of `engine/state_cache.py` over it."""
from __future__ import annotations

import torch

ALIGN = 32     # elements: 128 bytes


class RecurrentStates:
    def __init__(self):
        self.row_elems = 0
        self._at = {}
        self.buf = self.snap = self.host = None

    def reserve(self, key, n: int):
        self._at[key] = (self.row_elems, int(n))
        self.row_elems += -(-int(n) // ALIGN) * ALIGN

    def allocate(self, rows: int, device, snapshot_slots: int = 0):
        n = max(self.row_elems, ALIGN)
        self.buf = torch.zeros((rows, n), dtype=torch.float32, device=device)
        self.snap = torch.zeros((snapshot_slots, n), dtype=torch.float32, device=device) if snapshot_slots > 0 else None

    def view(self, key) -> torch.Tensor:
        off, n = self._at[key]
        return self.buf[:, off:off + n]

    def bytes_per_row(self) -> int:
        return self.row_elems * 4


class RecurrentStateMixin:
    """Expects `self.states` (RecurrentStates) with its buffers allocated."""

    supports_prefix_cache = False        # a shared prefix needs the state at its end: snapshots decide

    @property
    def state_snapshot_slots(self) -> int:
        return 0 if self.states.snap is None else self.states.snap.shape[0]

    def save_state_snapshot(self, slot: int, req_idx: int):
        self.states.snap[slot].copy_(self.states.buf[req_idx])

    def load_state_snapshot(self, slot: int, req_idx: int):
        self.states.buf[req_idx].copy_(self.states.snap[slot])

    def alloc_host_snapshots(self, nbytes: int) -> int:
        k = int(nbytes) // max(self.states.snap.shape[1] * 4, 1)
        if k <= 0:
            return 0
        self.states.host = torch.empty((k, self.states.snap.shape[1]), dtype=torch.float32,
                                       pin_memory=self.device.type == "cuda")
        return k

    def export_state_snapshot(self, slot: int, host_slot: int):
        self.states.host[host_slot].copy_(self.states.snap[slot])      # synchronous: the slot is used again right after

    def import_state_snapshot(self, host_slot: int, slot: int):
        self.states.snap[slot].copy_(self.states.host[host_slot], non_blocking=True)

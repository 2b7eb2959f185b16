"""Per-sequence recurrent state beside the KV caches.

One `RecurrentState` serves all layers of a model: for every array a layer registers it holds a device tensor
[slots, ...] in fp32.  A live sequence owns one slot for its whole life; rows are kept in the same order as the rows of
the layers' `Attention` caches, so `ModelHost` treats it like one more cache (`remove_seq`, `clear`, `duplicate`).
Slots are handed out lowest first and used again without being cleared: the kernels take a state as zero when a
sequence is at position 0.
"""
import bisect

import torch


class RecurrentState:
    def __init__(self, device, slots=16):
        self.device = torch.device(device)
        self.capacity = max(1, slots)
        self.arrays = {}
        self.rows = []       # slot of each live sequence, in row order
        self.length = {}     # slot -> tokens the sequence has run
        self.free = list(range(self.capacity))
        self.views = []      # per-layer handles into the caches, where a model's layers share caches

    def register(self, name, shape):
        """An array of per-sequence state; read it back with state[name] (it moves when the slots grow)."""
        self.arrays[name] = torch.zeros((self.capacity,) + tuple(shape), dtype=torch.float32, device=self.device)

    def __getitem__(self, name):
        return self.arrays[name]

    def __len__(self):
        return len(self.rows)

    def bytes_per_slot(self):
        return sum(a[0].numel() * 4 for a in self.arrays.values())

    def _grow(self):
        self.free.extend(range(self.capacity, 2 * self.capacity))
        for name, a in self.arrays.items():
            self.arrays[name] = torch.cat([a, torch.zeros_like(a)])
        self.capacity *= 2

    def insert(self, row):
        """A new sequence at row `row`; the rows after it move up."""
        if not 0 <= row <= len(self.rows):
            raise IndexError("row %d outside [0, %d]" % (row, len(self.rows)))
        if not self.free:
            self._grow()
        slot = self.free.pop(0)
        self.rows.insert(row, slot)
        self.length[slot] = 0
        return slot

    def remove_seq(self, row):
        slot = self.rows.pop(row)
        del self.length[slot]
        bisect.insort(self.free, slot)

    def duplicate(self, row, copies):
        """Clones of row `row` as the rows right after it (the row order of `Attention.duplicate`)."""
        src = self.rows[row]
        for c in range(copies):
            dst = self.insert(row + 1 + c)
            for a in self.arrays.values():
                a[dst].copy_(a[src])
            self.length[dst] = self.length[src]

    def clear(self):
        for row in reversed(range(len(self.rows))):
            self.remove_seq(row)

"""Per-sequence state on the device: slots that hold everything a sequence carries from step to step.

A layer reserves what it needs per sequence -- a recurrent state, the last inputs of a convolution, the ring of cached rows of a
sliding window -- and gets back a handle with slot 0's address and the stride between slots.  All reservations of a slot lie in one
record, so opening a sequence clears it with one memset; rows that are addressed by position and masked by it (rings) live in a
second record that needs no clearing.  The position of a slot's next token and its last token are device words, so a recorded
step serves every position and every set of slots.
"""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import native as N
from .device import Device, _SIZE

_ALIGN = 256


class Reservation:
    """ptr: slot 0's address; stride: elements between slots."""

    def __init__(self, arena: int, offset: int, dtype: int):
        self.arena, self.offset, self.dtype = arena, offset, dtype
        self.ptr = self.stride = 0


class SequenceStates:
    def __init__(self, dev: Device, slots: int):
        self.dev, self.slots = dev, slots
        self._bytes = [0, 0]                    # record sizes: cleared when a sequence opens / not
        self._reserved: list[Reservation] = []
        self._free = list(range(slots - 1, -1, -1))
        self.position: dict[int, int] = {}      # host mirror of `pos` for the open slots
        self.blocks = None
        self.pos = dev.zeros(slots, N.NS_I32)
        self.last = dev.zeros(slots, N.NS_I32)

    def reserve(self, count: int, dtype: int, cleared: bool) -> Reservation:
        assert self.blocks is None, "reservations end with allocate()"
        arena = 0 if cleared else 1
        r = Reservation(arena, self._bytes[arena], dtype)
        self._bytes[arena] += (count * _SIZE[dtype] + _ALIGN - 1) // _ALIGN * _ALIGN
        self._reserved.append(r)
        return r

    def allocate(self) -> None:
        self.blocks = [self.dev.empty(max(1, self.slots * n), N.NS_I8) for n in self._bytes]
        for r in self._reserved:
            r.ptr = self.blocks[r.arena].ptr + r.offset
            r.stride = self._bytes[r.arena] // _SIZE[r.dtype]

    @property
    def bytes_per_sequence(self) -> int:
        return sum(self._bytes)

    def open(self) -> int:
        """A slot at position 0 with everything in it cleared."""
        if not self._free:
            raise RuntimeError(f"all {self.slots} sequence slots are in use")
        slot = self._free.pop()
        self.rewind(slot)
        return slot

    def rewind(self, *slots: int) -> None:
        """Back to position 0, everything cleared; neighbouring slots are cleared together."""
        h, order = self.dev.handle, sorted(slots)
        at = 0
        while at < len(order):
            n = 1
            while at + n < len(order) and order[at + n] == order[at] + n:
                n += 1
            first = order[at]
            if self._bytes[0]:
                N.call("ns_memset32_async", h, C.c_uint64(self.blocks[0].ptr + first * self._bytes[0]), 0, C.c_uint64(n * self._bytes[0] // 4))
            N.call("ns_memset32_async", h, C.c_uint64(self.pos.ptr + 4 * first), 0, C.c_uint64(n))
            N.call("ns_memset32_async", h, C.c_uint64(self.last.ptr + 4 * first), 0xFFFFFFFF, C.c_uint64(n))
            at += n
        for s in slots:
            self.position[s] = 0

    def close(self, slot: int) -> None:
        del self.position[slot]
        self._free.append(slot)

"""What the sequences being generated hold on the device, for every model alike.

A model lists its parts: ``rows`` parts grow with the sequence (a KV or latent cache, room for ``capacity``
tokens, or for the latest ``limit`` of them where no token looks further back) and ``fixed`` parts do not
(recurrent states, convolution windows; zero at the start of a sequence).  :class:`SequenceSlots` owns one device block with a slot per live sequence; a slot that is
given back is used again by the next sequence.
"""
from dataclasses import dataclass

from . import capi

ALIGN = 256


@dataclass(frozen=True)
class StatePart:
    name: str
    nbytes: int              # of one token for rows, of the whole part for fixed
    rows: bool = False
    zero: bool = True        # cleared when a sequence starts (cache rows that are never read before they are written need not be)
    limit: int = 0           # most rows that are kept (token i in row i mod limit); 0: all

    def count(self, capacity):
        """Rows of the part in a slot."""
        return (min(capacity, self.limit) if self.limit else capacity) if self.rows else 1

    def size(self, capacity):
        n = self.nbytes * self.count(capacity)
        return -(-n // ALIGN) * ALIGN


@dataclass(frozen=True)
class StateLayout:
    offsets: dict
    slot_bytes: int


def lay_out(parts, capacity):
    """Byte offset of every part inside a slot; the parts to be cleared come first, back to back."""
    offsets, at = {}, 0
    for part in sorted(parts, key=lambda p: not p.zero):
        offsets[part.name] = at
        at += part.size(capacity)
    return StateLayout(offsets, max(at, ALIGN))


class Sequence:
    """One live sequence: its slot's device address and how many tokens it holds."""

    def __init__(self, slot, base, capacity):
        self.slot, self.base, self.capacity, self.length = slot, base, capacity, 0


class SequenceSlots:
    def __init__(self, lib, parts, capacity, slots=1, stream=None):
        if capacity < 1 or slots < 1:
            raise ValueError("capacity and slots start at 1")
        self.lib, self.capacity, self.stream = lib, capacity, stream
        self.parts = list(parts)
        self.layout = lay_out(self.parts, capacity)
        self.zero_bytes = sum(p.size(capacity) for p in self.parts if p.zero)
        self.block = lib.bpdq_alloc(self.layout.slot_bytes * slots)
        if not self.block:
            raise MemoryError(f"device allocation of {self.layout.slot_bytes * slots} bytes for {slots} sequences failed")
        self.free = list(range(slots))

    def acquire(self):
        """A fresh sequence, or None when every slot is in use."""
        if not self.free:
            return None
        slot = self.free.pop(0)
        seq = Sequence(slot, self.block + slot * self.layout.slot_bytes, self.capacity)
        if self.zero_bytes:
            capi.check(self.lib.bpdq_memset_async(seq.base, 0, self.zero_bytes, self.stream), "clearing a sequence's state")
        return seq

    def release(self, seq):
        if seq.slot is None:
            raise ValueError("the sequence has been released already")
        self.free.append(seq.slot)
        seq.slot = None

    def address(self, seq, name):
        return seq.base + self.layout.offsets[name]

    def close(self):
        if self.block:
            self.lib.bpdq_free(self.block)
            self.block = None

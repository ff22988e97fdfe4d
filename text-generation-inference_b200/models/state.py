"""Pools a shard hands out to requests: pages of the KV cache and slots of the recurrent state.

A request's KV pages come from the router (``router/src/radix.hpp``); its recurrent state is the shard's own
business: one slot per live request, held from the first step that brings its tokens until the request leaves its
batch.  A slot is never cleared: a sequence whose step starts at position 0 starts from a zero state in the kernels.
"""
from __future__ import annotations

from typing import List


class Pool:
    """Fixed set of numbered units, handed out last-returned-first."""

    def __init__(self, first: int, count: int, what: str):
        self.capacity, self.what = count, what
        self._free: List[int] = list(range(first + count - 1, first - 1, -1))

    @property
    def available(self) -> int:
        return len(self._free)

    def take(self) -> int:
        if not self._free:
            raise RuntimeError(f"out of {self.what}: all {self.capacity} are held by live requests")
        return self._free.pop()

    def give(self, unit: int) -> None:
        self._free.append(unit)


class Lease:
    """One unit of a pool; returned by ``release`` or, for holders that are simply dropped, with the object."""

    __slots__ = ("pool", "unit")

    def __init__(self, pool: Pool):
        self.unit = None
        self.pool = pool
        self.unit = pool.take()

    def release(self) -> None:
        if self.unit is not None:
            self.pool.give(self.unit)
            self.unit = None

    def __del__(self):
        self.release()

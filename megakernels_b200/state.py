"""Per-sequence state of a model: slots, key/value rows and recurrent matrices.

A slot is one sequence's share of every cache.  ``SlotPool`` hands slots out and takes them back;
``HybridState`` owns the tensors of a layer-list model (``hybrid.py``):

* attention layers that project their own keys and values hold ``keep + ring`` rows per slot: the
  first ``keep`` positions for good, later positions modulo ``ring``.  Layers that read another
  layer's rows own nothing; ``keep`` and ``ring`` cover the widest reader;
* recurrent layers hold one 32-bit matrix per head and slot, value column by value column.

Nothing has to be cleared between owners of a slot: a sequence starts at position 0, where the
kernels take the recurrent state as zero, and no query looks at a position that its own sequence
has not written.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import Tensor


class SlotPool:
    """Free list of ``count`` slots; the slot freed last is handed out first."""

    def __init__(self, count: int):
        self.count = count
        self._free = list(range(count - 1, -1, -1))
        self._used: set[int] = set()

    def allocate(self) -> int:
        if not self._free:
            raise RuntimeError(f"all {self.count} sequence slots are in use")
        slot = self._free.pop()
        self._used.add(slot)
        return slot

    def free(self, slot: int) -> None:
        if slot not in self._used:
            raise ValueError(f"slot {slot} is not in use")
        self._used.remove(slot)
        self._free.append(slot)

    def __len__(self) -> int:
        return len(self._used)


@dataclass(frozen=True)
class CacheRows:
    """Geometry of one layer's key/value rows."""

    keep: int
    ring: int

    @property
    def total(self) -> int:
        return self.keep + self.ring

    def row(self, position: int) -> int:
        """Row of a position (the kernels' ``cache_row``)."""
        return position if position < self.keep else self.keep + (position - self.keep) % self.ring


def plan_cache_rows(readers: list, max_len: int, portion: int) -> CacheRows:
    """Rows that serve every reader (objects with ``window`` and ``keep_first``) of one cache.

    A portion of ``portion`` tokens is written before its first token attends, so a ring of
    ``window + portion`` rows never overwrites a visible position.  A sequence shorter than that
    gets one row per position.
    """
    keep = min(max(r.keep_first for r in readers), max_len)
    ring = max(1, min(max(r.window for r in readers) + portion, max_len - keep))
    return CacheRows(keep, ring)


class HybridState:
    def __init__(self, config, slots: int, max_len: int, portion: int, device, dtype: torch.dtype):
        self.pool = SlotPool(slots)
        self.rows: dict[int, CacheRows] = {}
        self.keys: dict[int, Tensor] = {}
        self.values: dict[int, Tensor] = {}
        self.matrices: dict[int, Tensor] = {}
        for i, layer in enumerate(config.layers):
            m = layer.mixer
            if m.kind == "delta_rule":
                self.matrices[i] = torch.zeros(slots, m.heads, m.dim, m.dim, device=device, dtype=torch.float32)
            elif m.kv_from is None:
                readers = [m] + [o.mixer for o in config.layers if getattr(o.mixer, "kv_from", None) == i]
                rows = self.rows[i] = plan_cache_rows(readers, max_len, portion)
                self.keys[i] = torch.zeros(slots, rows.total, m.kv_heads, 2, m.dim, device=device, dtype=dtype)
                self.values[i] = torch.zeros(slots, rows.total, m.kv_heads, m.vdim, device=device, dtype=dtype)

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size()
                   for d in (self.keys, self.values, self.matrices) for t in d.values())

"""Per-sequence state of a model: slots, key/value rows and recurrent matrices.

A slot is one sequence's share of every cache.  ``SlotPool`` hands slots out and takes them back;
``HybridState`` owns the tensors of a layer-list model (``hybrid.py``):

* attention layers that project their own keys and values hold ``keep + ring`` rows per slot: the
  first ``keep`` positions for good, later positions modulo ``ring``.  Layers that read another
  layer's rows own nothing; ``keep`` and ``ring`` cover the widest reader.  A latent attention's row
  is the latent and the rotated key part;
* recurrent layers hold one 32-bit matrix per head and slot, value column by value column;
* a convolution over time of ``taps`` holds its last ``taps - 1`` inputs in a ring by position, and
  the sum of the terms that they add to the next position (32-bit).

Keys of the dictionaries are layer runs: each pass of a loop has its own.  Nothing has to be cleared
between owners of a slot: a sequence starts at position 0, where the kernels take the recurrent
state and earlier inputs as zero, and no query looks at a position that its own sequence has not
written.
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
        self.inputs: dict[int, Tensor] = {}  # input convolution: [slots, taps - 1, width]
        self.input_terms: dict[int, Tensor] = {}  # [slots, 2, width], in turn by the position's parity
        self.projected: dict[int, Tensor] = {}  # the projections' convolution: [slots, taps - 1, rows]
        self.projected_terms: dict[int, Tensor] = {}  # [slots, rows]
        layers = config.run_layers
        f32 = lambda *shape: torch.zeros(slots, *shape, device=device, dtype=torch.float32)  # noqa: E731
        for i, layer in enumerate(layers):
            m = layer.mixer
            if m.kind == "delta_rule":
                self.matrices[i] = f32(m.heads, m.dim, m.dim)
            elif m.kv_from is None:
                readers = [m] + [o.mixer for o in layers if getattr(o.mixer, "kv_from", None) == i]
                rows = self.rows[i] = plan_cache_rows(readers, max_len, portion)
                if m.kind == "latent_attention":
                    self.keys[i] = torch.zeros(slots, rows.total, m.row_elems, device=device, dtype=dtype)
                elif m.kind == "attention":  # (a head's rows together: its splits are runs of memory)
                    cache = lambda n: torch.zeros(slots, m.kv_heads, rows.total, n, device=device, dtype=dtype)  # noqa: E731
                    self.keys[i], self.values[i] = cache(m.dim), cache(m.vdim)
                else:
                    cache = lambda *shape: torch.zeros(slots, rows.total, m.kv_heads, *shape, device=device, dtype=dtype)  # noqa: E731
                    self.keys[i], self.values[i] = cache(2, m.dim), cache(m.vdim)
            if layer.canon_taps:
                self.inputs[i], self.input_terms[i] = f32(max(layer.canon_taps - 1, 1), config.width), f32(2, config.width)
            if getattr(m, "conv_taps", 0):
                self.projected[i], self.projected_terms[i] = f32(max(m.conv_taps - 1, 1), m.in_rows), f32(m.in_rows)

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size()
                   for d in (self.keys, self.values, self.matrices, self.inputs, self.input_terms, self.projected, self.projected_terms)
                   for t in d.values())

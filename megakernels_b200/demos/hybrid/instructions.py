"""Decode instruction set of layer-list models and the globals its kernels run on.

Same encoding as the latency set (``Instruction.serialize``): opcode, then the fields.  One
instruction covers a run of whole output rows (projections), a block of value columns of one
recurrence head, or one split of the visible keys of a KV head; the phases of a layer are ordered
by one arrival counter per layer and opcode.
"""

from __future__ import annotations

from dataclasses import dataclass, field

import torch
from torch import Tensor

from megakernels_b200.instructions import Instruction
from megakernels_b200.utils import get_sm_count

COUNTERS_PER_LAYER = 12  # MKBH_BARRIERS_PER_LAYER
MAX_ROWS = 512  # output rows of an instruction
PARTIAL_SUMS = 4096  # per-row, per-column-group sums an instruction may hold


@dataclass
class HybridGlobals:
    """Everything a launch reads or writes; prefill and decode share the activation buffers."""

    model: object
    device: torch.device
    portion: int

    tokens: Tensor  # int32 [portion]
    want_rows: Tensor  # int32 [portion]
    x: Tensor  # fp32 [portion (decode: 2), width]: the residual stream
    proj: Tensor  # fp32 [portion, stacked projection rows or ff]
    mixed: Tensor  # fp32 [portion, mixer output]
    decay: Tensor  # fp32 [portion, recurrence channels]
    act: Tensor  # model dtype [portion, widest matrix input]
    logits: Tensor  # fp32 [vocab]
    argmax_out: Tensor  # int32 [1]
    counters: Tensor  # int32, zeroed by every decode launch
    arrivals: Tensor  # int32 [layer runs + 1, COUNTERS_PER_LAYER]
    attn_part: Tensor  # fp32 [max heads, 2, max_splits, 4 + max vdim]
    status: Tensor  # int32 [16]
    max_splits: int
    max_kv_heads: int
    part_vdim: int
    query: Tensor  # model dtype [portion, heads * query/key size]: rotated queries
    act2: Tensor  # model dtype [portion, width]: input of a feed-forward beside a mixer
    ffn: Tensor  # model dtype [portion, ff]: gated units
    keys: Tensor  # model dtype [positions, heads * (dim + vdim)]: keys and values expanded from latents
    tail: Tensor  # fp32 [taps, width]: the portion's last inputs of the input convolution
    side: Tensor  # fp32 [side_ff + width + side_rank]: decode vectors beside the stacked projection
    side_ff: int
    side_rank: int

    slot: int = 0
    pos_id: int = 0
    pos_id_device: Tensor | None = None  # int32 [1]; overrides pos_id in decode launches
    instructions: Tensor | None = None
    timings: Tensor | None = None
    hooks: dict = field(default_factory=dict)

    def sm_count(self) -> int:
        return get_sm_count(self.device)

    @property
    def dtype_bytes(self) -> int:
        return 4 if self.model.dtype == torch.float32 else 2


def matrix_shape(globs: HybridGlobals, opcode: int, layer: int) -> tuple[int, int]:
    """(rows, input columns) of the matrix an instruction streams."""
    cfg = globs.model.config
    if opcode == Head.opcode():
        return cfg.vocab_size, cfg.width
    spec = cfg.run_layers[layer]
    m, mlp = spec.mixer, spec.mlp
    if opcode == Enter.opcode():
        return cfg.width, 2 * cfg.width
    if opcode == Absorb.opcode():
        return m.heads * m.rank, m.dim
    if opcode == Expand.opcode():
        return m.out_features, m.rank
    return {
        NormProj.opcode(): (m.in_rows, cfg.width),
        OutProj.opcode(): (cfg.width, m.out_features),
        NormUp.opcode(): (mlp.up_rows if mlp else 0, cfg.width),
        Down.opcode(): (cfg.width, mlp.ff if mlp else 0),
    }[opcode]


@dataclass
class RowRange(Instruction):
    layer_idx: int
    row_start: int
    row_end: int

    @classmethod
    def tags(cls):
        return {"pool": "memory"}

    def cost(self, globs) -> float:
        return (self.row_end - self.row_start) * matrix_shape(globs, self.opcode(), self.layer_idx)[1]


@dataclass
class NormProj(RowRange):
    """Norm of the residual stream, input convolution, stacked input projection of the mixer."""

    @classmethod
    def opcode(cls) -> int:
        return 1


@dataclass
class DeltaStep(Instruction):
    """One step of a head's recurrence for value columns ``[col_start, col_end)``."""

    layer_idx: int
    head_idx: int
    col_start: int
    col_end: int

    @classmethod
    def opcode(cls) -> int:
        return 2

    @classmethod
    def tags(cls):
        return {"pool": "compute"}

    def cost(self, globs) -> float:
        m = globs.model.config.run_layers[self.layer_idx].mixer
        return (self.col_end - self.col_start) * m.dim * 4


@dataclass
class KeyAttention(Instruction):
    """One split of the keys that a KV head's queries see; the last split to arrive merges them (of a
    latent: ``Expand`` does)."""

    layer_idx: int
    kv_head_idx: int
    split_idx: int
    num_splits: int

    @classmethod
    def opcode(cls) -> int:
        return 3

    @classmethod
    def tags(cls):
        return {"pool": "compute"}

    def cost(self, globs) -> float:
        m = globs.model.config.run_layers[self.layer_idx].mixer
        return min(m.window + m.keep_first, globs.model.max_len()) * m.key_elems / m.key_groups / self.num_splits


@dataclass
class OutProj(RowRange):
    """Output projection of the mixer, layer scale, residual add."""

    @classmethod
    def opcode(cls) -> int:
        return 4


@dataclass
class NormUp(RowRange):
    """Norm, up projection of the feed-forward (with a gate: the gated unit)."""

    @classmethod
    def opcode(cls) -> int:
        return 5


@dataclass
class Down(RowRange):
    """Activation, down projection, layer scale, residual add (beside a mixer: left to ``OutProj``)."""

    @classmethod
    def opcode(cls) -> int:
        return 6


@dataclass
class Head(RowRange):
    """Final norm, logits and their running argmax."""

    @classmethod
    def opcode(cls) -> int:
        return 7


@dataclass
class Enter(RowRange):
    """Start of a pass of the loop: the residual stream and the embedding, projected to one stream."""

    @classmethod
    def opcode(cls) -> int:
        return 8


@dataclass
class Absorb(RowRange):
    """Latent attention: a head's query times the key expansion (rows of one head)."""

    @classmethod
    def opcode(cls) -> int:
        return 9


@dataclass
class Expand(RowRange):
    """Latent attention: a head's output, merged over the splits of the keys, from latent to value
    space (rows of one head)."""

    num_splits: int

    @classmethod
    def opcode(cls) -> int:
        return 10

"""Schedule builder of layer-list models: one token as a DAG of instructions.

Every phase of a layer is spread over all SMs (rows of a projection, column blocks of a
recurrence, key splits of an attention); a phase depends on the whole phase before it.  In a layer
whose feed-forward runs beside the mixer, the feed-forward's instructions fill the queues where the
mixer's next phase would wait for the previous one.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from megakernels_b200.demos.hybrid.instructions import (
    COUNTERS_PER_LAYER,
    MAX_ROWS,
    PARTIAL_SUMS,
    Absorb,
    DeltaStep,
    Down,
    Enter,
    Expand,
    Head,
    HybridGlobals,
    NormProj,
    NormUp,
    OutProj,
    KeyAttention,
    matrix_shape,
)
from megakernels_b200.hybrid import key_splits, pad8
from megakernels_b200.scheduler import DAG_Node, ScheduleBuilder


@dataclass
class HybridScheduleOptions:
    keys_per_split: int = 64  # visible keys per attention instruction, about
    state_columns: int = 0  # value columns per recurrence instruction (0: from the SM count)


def column_groups(in_features: int, elem_bytes: int) -> int:
    """Consumer warps that share a weight row (the kernel's ``column_groups``)."""
    chunks = pad8(in_features) * elem_bytes // 16
    n = 1
    while n < 16 and n * 32 < chunks:
        n *= 2
    return n


def row_ranges(rows: int, in_features: int, elem_bytes: int, sm_count: int, unit: int = 1) -> list[tuple[int, int]]:
    """Contiguous runs of rows, as even as possible: one per SM, or the fewest equal waves whose
    runs fit the partial-sum buffer.  ``unit`` rows stay together."""
    most = min(MAX_ROWS, PARTIAL_SUMS // column_groups(in_features, elem_bytes)) // unit
    rows //= unit
    count = min(rows, sm_count * -(-rows // (sm_count * most)))
    return [(rows * i // count * unit, rows * (i + 1) // count * unit) for i in range(count)]


def state_columns(heads: int, dim: int, sm_count: int) -> int:
    """Columns per recurrence instruction (a warp carries one at a time, 16 side by side): the
    narrowest block that fits one wave of SMs."""
    c = 16
    while c < dim and heads * -(-dim // c) > sm_count:
        c += 16
    return c


def head_row_ranges(heads: int, rows: int, in_features: int, elem_bytes: int, sm_count: int) -> list[tuple[int, int]]:
    """Rows of a block-diagonal product, ``rows`` per head; a run stays within a head."""
    one = row_ranges(rows, in_features, elem_bytes, max(1, sm_count // heads))
    return [(h * rows + a, h * rows + b) for h in range(heads) for a, b in one]


def make_globals(model, options: HybridScheduleOptions) -> HybridGlobals:
    cfg, device, n = model.config, model.device, model.portion()
    layers = cfg.layers
    attn = [s.mixer for s in layers if s.mixer.kind != "delta_rule"]
    delta = [s.mixer for s in layers if s.mixer.kind == "delta_rule"]
    latent = [s.mixer for s in layers if s.mixer.kind == "latent_attention"]
    rotary = [s.mixer for s in layers if s.mixer.kind == "attention"]
    poly = [s.mlp.ff for s in layers if s.mlp is not None and s.mlp.kind == "poly_norm"]
    glu = [s.mlp.ff for s in layers if s.mlp is not None and s.mlp.kind == "clamped_glu"]
    widest = lambda sizes: max([pad8(x) for x in sizes], default=0)  # noqa: E731
    pad64 = lambda x: -(-x // 64) * 64  # noqa: E731  (whole tensor-core slabs per query head)
    mixed = widest(s.mixer.out_features for s in layers)
    act = max(widest([cfg.width * (2 if cfg.loop else 1)]), mixed, widest(poly))
    from megakernels_b200.utils import get_sm_count

    sms = get_sm_count(device)
    splits = max([key_splits(a, model.max_len(), sms, options.keys_per_split) for a in attn], default=1)
    groups = max([a.key_groups for a in attn], default=1)
    vdim = max([a.rank if a.kind == "latent_attention" else a.vdim for a in attn], default=1)
    heads = max([a.heads for a in attn], default=1)
    f32 = lambda *shape: torch.zeros(shape, device=device, dtype=torch.float32)  # noqa: E731
    i32 = lambda *shape: torch.zeros(shape, device=device, dtype=torch.int32)  # noqa: E731
    own = lambda *shape: torch.zeros(shape, device=device, dtype=model.dtype)  # noqa: E731
    R = len(cfg.runs)
    side_ff, side_rank = widest(glu), widest(m.heads * m.rank for m in latent)
    return HybridGlobals(
        model=model, device=device, portion=n,
        tokens=i32(n), want_rows=i32(n), x=f32(max(n, 2), cfg.width),
        proj=f32(n, max(widest(s.mixer.in_rows for s in layers), widest(poly))), mixed=f32(n, mixed),
        decay=f32(n, max([d.inner + 2 * d.heads for d in delta], default=1)), act=own(n, act),
        logits=f32(cfg.vocab_size), argmax_out=i32(1),
        counters=i32((2 + (R + 1) * COUNTERS_PER_LAYER + R * groups + 1) // 2 * 2),
        arrivals=i32(R + 1, COUNTERS_PER_LAYER), attn_part=f32(heads, 2, splits, 4 + -(-vdim // 4) * 4), status=i32(16),
        max_splits=splits, max_kv_heads=groups, part_vdim=vdim,
        query=own(n, max([m.heads * (pad64(m.dim) + pad64(m.rot_dim)) for m in latent] + [m.heads * pad64(m.dim) for m in rotary] + [1])),
        act2=own(n, widest([cfg.width])), ffn=own(n, max(side_ff, 1)),
        keys=own(model.max_len(), widest(m.heads * (m.dim + m.vdim) for m in latent)) if latent else own(1),
        tail=f32(max([s.canon_taps for s in layers] + [1]), cfg.width), side=f32(side_ff + pad8(cfg.width) + side_rank),
        side_ff=side_ff, side_rank=side_rank,
    )


class HybridScheduleBuilder(ScheduleBuilder):
    def __init__(self, options: HybridScheduleOptions | None = None):
        self.options = options or HybridScheduleOptions()

    def make_globals(self, model):
        return make_globals(model, self.options)

    def make_dag(self, globs: HybridGlobals, stop_after_op=None, layer_limit=None):
        if stop_after_op is not None:
            raise ValueError("stop_after_op is not available for layer-list models")
        cfg, sms = globs.model.config, globs.sm_count()
        nodes: list[DAG_Node] = []
        arrivals = torch.zeros(globs.arrivals.shape, dtype=torch.int32)

        def phase(instructions, previous, counter_layer, arrive=None):
            now = [DAG_Node(ins, list(previous)) for ins in instructions]
            nodes.extend(now)
            arrivals[counter_layer, instructions[0].opcode()] = len(now) if arrive is None else arrive
            return now

        def rows(cls, layer, unit=1):
            n, k = matrix_shape(globs, cls.opcode(), layer)
            return [cls(layer, a, b) for a, b in row_ranges(n, k, globs.dtype_bytes, sms, unit)]

        def head_rows(cls, layer, heads, *rest):
            n, k = matrix_shape(globs, cls.opcode(), layer)
            return [cls(layer, a, b, *rest) for a, b in head_row_ranges(heads, n // heads, k, globs.dtype_bytes, sms)]

        def up(i, spec, previous):
            return phase(rows(NormUp, i, unit=2 if spec.mlp.kind == "clamped_glu" else 1), previous, i)

        last: list[DAG_Node] = []
        for i, (layer, enters) in enumerate(cfg.runs[:layer_limit]):
            spec = cfg.layers[layer]
            m, beside = spec.mixer, spec.parallel and spec.mlp is not None
            if enters:
                last = phase(rows(Enter, i), last, i)
            before = last
            last = phase(rows(NormProj, i), before, i)
            inner = up(i, spec, before) if beside else []
            if m.kind == "delta_rule":
                c = self.options.state_columns or state_columns(m.heads, m.dim, sms)
                steps = [DeltaStep(i, h, a, min(a + c, m.dim)) for h in range(m.heads) for a in range(0, m.dim, c)]
                last = phase(steps, last, i)
            else:
                if m.kind == "latent_attention":
                    last = phase(head_rows(Absorb, i, m.heads), last, i)
                n = key_splits(m, globs.model.max_len(), sms, self.options.keys_per_split)
                splits = [KeyAttention(i, g, s, n) for g in range(m.key_groups) for s in range(n)]
                last = phase(splits, last, i, arrive=None if m.kind == "latent_attention" else m.key_groups)
            down = phase(rows(Down, i), inner, i) if beside else []
            if m.kind == "latent_attention":
                last = phase(head_rows(Expand, i, m.heads, n), last, i)
            # (beside a mixer, ``Down`` counts into the phase that ``OutProj`` waits for)
            arrivals[i, last[0].instruction.opcode()] += len(down)
            last = phase(rows(OutProj, i), last + down, i)
            if spec.mlp is not None and not beside:
                last = up(i, spec, last)
                last = phase(rows(Down, i), last, i)
        last = phase(rows(Head, 0), last, len(cfg.runs))
        globs.arrivals.copy_(arrivals)
        end = DAG_Node(nodes[-1].instruction, last)
        return nodes, end

    def build(self, model, stop_after_op=None, layer_limit=None):
        from megakernels_b200.scheduler import Schedule

        globs = self.make_globals(model)
        nodes, end = self.make_dag(globs, stop_after_op, layer_limit)
        return Schedule(globs, nodes, end)

"""Schedule builder of layer-list models: one token as a DAG of instructions.

Every phase of a layer is spread over all SMs (rows of a projection, column blocks of a
recurrence, key splits of an attention); a phase depends on the whole phase before it.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from megakernels_b200.demos.hybrid.instructions import (
    COUNTERS_PER_LAYER,
    MAX_ROWS,
    PARTIAL_SUMS,
    DeltaStep,
    Down,
    Head,
    HybridGlobals,
    NormProj,
    NormUp,
    OutProj,
    WindowAttention,
    matrix_shape,
)
from megakernels_b200.hybrid import pad8
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


def row_ranges(rows: int, in_features: int, elem_bytes: int, sm_count: int) -> list[tuple[int, int]]:
    """Contiguous runs of rows, as even as possible: one per SM, or the fewest equal waves whose
    runs fit the partial-sum buffer."""
    most = min(MAX_ROWS, PARTIAL_SUMS // column_groups(in_features, elem_bytes))
    count = min(rows, sm_count * -(-rows // (sm_count * most)))
    return [(rows * i // count, rows * (i + 1) // count) for i in range(count)]


def state_columns(heads: int, dim: int, sm_count: int) -> int:
    """Columns per recurrence instruction (a warp carries one at a time, 16 side by side): the
    narrowest block that fits one wave of SMs."""
    c = 16
    while c < dim and heads * -(-dim // c) > sm_count:
        c += 16
    return c


def make_globals(model, options: HybridScheduleOptions) -> HybridGlobals:
    cfg, device, n = model.config, model.device, model.portion()
    attn = [s.mixer for s in cfg.layers if s.mixer.kind == "diff_attention"]
    delta = [s.mixer for s in cfg.layers if s.mixer.kind == "delta_rule"]
    ffs = [s.mlp.ff for s in cfg.layers if s.mlp is not None]
    proj = max([pad8(s.mixer.in_rows) for s in cfg.layers] + [pad8(f) for f in ffs])
    mixed = max(pad8(s.mixer.out_features) for s in cfg.layers)
    act = max([pad8(cfg.width), mixed] + [pad8(f) for f in ffs])
    from megakernels_b200.utils import get_sm_count

    sms = get_sm_count(device)
    splits = max([a.num_splits(sms, options.keys_per_split) for a in attn], default=1)
    kv_heads = max([a.kv_heads for a in attn], default=1)
    vdim = max([a.vdim for a in attn], default=1)
    heads = max([a.heads for a in attn], default=1)
    f32 = lambda *shape: torch.zeros(shape, device=device, dtype=torch.float32)  # noqa: E731
    i32 = lambda *shape: torch.zeros(shape, device=device, dtype=torch.int32)  # noqa: E731
    L = cfg.num_hidden_layers
    return HybridGlobals(
        model=model, device=device, portion=n,
        tokens=i32(n), want_rows=i32(n), x=f32(n, cfg.width), proj=f32(n, proj), mixed=f32(n, mixed),
        decay=f32(n, max([d.inner + 2 * d.heads for d in delta], default=1)),
        act=torch.zeros(n, act, device=device, dtype=model.dtype),
        logits=f32(cfg.vocab_size), argmax_out=i32(1),
        counters=i32((2 + (L + 1) * COUNTERS_PER_LAYER + L * kv_heads + 1) // 2 * 2),
        arrivals=i32(L + 1, COUNTERS_PER_LAYER), attn_part=f32(heads, 2, splits, vdim + 2), status=i32(16),
        max_splits=splits, max_kv_heads=kv_heads, part_vdim=vdim,
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

        def rows(cls, layer):
            n, k = matrix_shape(globs, cls.opcode(), layer)
            return [cls(layer, a, b) for a, b in row_ranges(n, k, globs.dtype_bytes, sms)]

        last: list[DAG_Node] = []
        for i, spec in enumerate(cfg.layers[:layer_limit]):
            m = spec.mixer
            last = phase(rows(NormProj, i), last, i)
            if m.kind == "delta_rule":
                c = self.options.state_columns or state_columns(m.heads, m.dim, sms)
                steps = [DeltaStep(i, h, a, min(a + c, m.dim)) for h in range(m.heads) for a in range(0, m.dim, c)]
                last = phase(steps, last, i)
            else:
                n = m.num_splits(sms, self.options.keys_per_split)
                splits = [WindowAttention(i, g, s, n) for g in range(m.kv_heads) for s in range(n)]
                last = phase(splits, last, i, arrive=m.kv_heads)
            last = phase(rows(OutProj, i), last, i)
            if spec.mlp is not None:
                last = phase(rows(NormUp, i), last, i)
                last = phase(rows(Down, i), last, i)
        last = phase(rows(Head, 0), last, cfg.num_hidden_layers)
        globs.arrivals.copy_(arrivals)
        end = DAG_Node(nodes[-1].instruction, last)
        return nodes, end

    def build(self, model, stop_after_op=None, layer_limit=None):
        from megakernels_b200.scheduler import Schedule

        globs = self.make_globals(model)
        nodes, end = self.make_dag(globs, stop_after_op, layer_limit)
        return Schedule(globs, nodes, end)

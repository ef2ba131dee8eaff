"""Mode name -> schedule builder / megakernel interpreter / generator.

Reference: megakernels/dispatch.py:17-42.  ``latency`` is the reference's setting (Llama);
``hybrid`` is the instruction set of layer-list models (``hybrid.py``).  The reference's
``throughput`` setting has no kernel in its own tree, and its Python VM is test
infrastructure that lives outside the product.
"""

from __future__ import annotations

from pathlib import Path

from megakernels_b200.demos.hybrid.mk import HybridMK_Interpreter
from megakernels_b200.demos.hybrid.scheduler import HybridScheduleBuilder, HybridScheduleOptions
from megakernels_b200.demos.latency.mk import LatencyMK_Interpreter
from megakernels_b200.demos.latency.scheduler import (
    LatencyScheduleBuilder,
    LatencyScheduleOptions,
)
from megakernels_b200.generators import Hybrid_Generator, MK_Generator
from megakernels_b200.mk import MK_Interpreter
from megakernels_b200.scheduler import ScheduleBuilder, assign_to_sms, tensorize_instructions

BUILDER_MAP = {"latency": LatencyScheduleBuilder, "hybrid": HybridScheduleBuilder}
MK_INTERPRETER_MAP = {"latency": LatencyMK_Interpreter, "hybrid": HybridMK_Interpreter}
GENERATOR_MAP = {"latency": MK_Generator, "hybrid": Hybrid_Generator}


def make_schedule_builder(
    mode: str, options: LatencyScheduleOptions | HybridScheduleOptions | None = None
) -> ScheduleBuilder:
    if mode not in BUILDER_MAP:
        raise KeyError(f"unknown setting {mode!r}; available: {sorted(BUILDER_MAP)}")
    return BUILDER_MAP[mode](options)


def make_mk_interpreter(mode: str, mk_dir: Path | None = None) -> MK_Interpreter:
    if mode not in MK_INTERPRETER_MAP:
        raise KeyError(f"unknown setting {mode!r}; available: {sorted(MK_INTERPRETER_MAP)}")
    return MK_INTERPRETER_MAP[mode](mk_dir)


def make_generator(
    model, options=None, sched: str = "rr", mk_dir: Path | None = None, memory_fraction: float | None = None, **kw
) -> MK_Generator:
    """Schedule, instruction queues, interpreter and generator of a model in one go."""
    mode = model.setting
    schedule = make_schedule_builder(mode, options).build(model)
    tensorize_instructions(schedule.globs, assign_to_sms(sched, schedule=schedule, memory_fraction=memory_fraction))
    return GENERATOR_MAP[mode](model, make_mk_interpreter(mode, mk_dir), schedule, **kw)


def make_pyvm_interpreter(mode: str):
    raise NotImplementedError(
        "the Python VM is a CPU checker, not a product path; it lives in oracle/python_vm.py "
        "and is only used by the tests"
    )

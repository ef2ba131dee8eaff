"""Bind ``HybridGlobals`` to the C ABI of the hybrid kernels."""

from __future__ import annotations

import torch

from megakernels_b200.demos.hybrid.instructions import HybridGlobals
from megakernels_b200.mk import MK_Interpreter


class HybridMK_Interpreter(MK_Interpreter):
    module_name = "mk_hybrid"

    def bind(self, globs: HybridGlobals):
        """The ctypes mirror of the globals; built once, refreshed per call."""
        call = globs.hooks.get("call")
        if call is None:
            call = globs.hooks["call"] = self.module.Call(globs)
        return call

    def interpret(self, globs: HybridGlobals, stream=None, record_timings: bool = False):
        """One token: ``globs.tokens[0]`` at ``globs.pos_id`` (or the device word) in ``globs.slot``."""
        call = self.bind(globs)
        call.decode(stream if stream is not None else torch.cuda.current_stream(globs.device), record_timings)
        return call

    def prefill(self, globs: HybridGlobals, num_tokens: int, num_want: int, logits, layers_out=None, stream=None):
        """``globs.tokens[:num_tokens]`` from ``globs.pos_id`` on; logits of ``want_rows[:num_want]``."""
        call = self.bind(globs)
        call.prefill(num_tokens, num_want, logits, layers_out,
                     stream if stream is not None else torch.cuda.current_stream(globs.device))
        return call

"""Which model class serves a checkpoint directory or a preset name."""

from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Callable

import torch

from megakernels_b200 import dumalix, torirax
from megakernels_b200.llama import LlamaConfig, LlamaForCausalLM
from megakernels_b200.model_types import ExtraModelConfig


@dataclass(frozen=True)
class ModelFamily:
    name: str
    model_class: type
    library: str  # native library its kernels live in (build.py)
    dtypes: tuple[torch.dtype, ...]
    matches: Callable[[dict], bool]  # parsed config.json -> is it this family
    presets: dict[str, Callable[..., Any]] = field(default_factory=dict)  # name -> random-weight configuration


FAMILIES = (
    ModelFamily(
        "torirax", torirax.ToriraxForCausalLM, "hybrid", (torch.bfloat16, torch.float32),
        lambda raw: raw.get("architecture") == "Torirax", dict(torirax.PRESETS),
    ),
    ModelFamily(
        "dumalix", dumalix.DumalixForCausalLM, "hybrid", (torch.bfloat16, torch.float32),
        lambda raw: raw.get("architecture") == "Dumalix", dict(dumalix.PRESETS),
    ),
    ModelFamily(
        "llama", LlamaForCausalLM, "llama", (torch.bfloat16,),
        lambda raw: "architecture" not in raw and "num_key_value_heads" in raw,
        {
            "llama-1b": LlamaConfig.llama_3_2_1b,
            "llama-8b": LlamaConfig.llama_3_1_8b,
            "llama-70b": LlamaConfig.llama_3_1_70b,
            "meta-llama/Llama-3.2-1B-Instruct": LlamaConfig.llama_3_2_1b,
            "meta-llama/Llama-3.1-8B-Instruct": LlamaConfig.llama_3_1_8b,
        },
    ),
)


def family_of_preset(name: str) -> ModelFamily | None:
    return next((f for f in FAMILIES if name in f.presets), None)


def family_of_checkpoint(path: str | Path) -> ModelFamily:
    raw = json.loads((Path(path) / "config.json").read_text())
    for f in FAMILIES:
        if f.matches(raw):
            return f
    raise ValueError(f"{path}: no model family for architecture {raw.get('architecture') or raw.get('architectures')!r}")


def load_model(
    path: str | Path,
    extra_config: ExtraModelConfig | None = None,
    device="cuda:0",
    dtype: torch.dtype = torch.bfloat16,
):
    """Model of a local checkpoint directory, its class chosen by ``config.json``."""
    family = family_of_checkpoint(path)
    if dtype not in family.dtypes:
        raise ValueError(f"{family.name} models do not run in {dtype}")
    return family.model_class.from_pretrained(path, extra_config, device=device, dtype=dtype)

"""Torirax: layer-list decoder of generalized-delta-rule and windowed differential-attention layers.

Reads a checkpoint directory (``config.json``, ``*.safetensors``) into the mechanisms of
``hybrid.py``.  Every size comes from the configuration or a tensor's shape; the decay's
``exp(-1/2)`` and the unit key's ``1e-6`` are constants of the design (defaults of
``DeltaRuleSpec``).
"""

from __future__ import annotations

import json
from pathlib import Path

import torch

from megakernels_b200.hybrid import (
    DeltaRuleSpec,
    DiffAttentionSpec,
    HybridConfig,
    HybridForCausalLM,
    LayerSpec,
    PolyNormSpec,
)
from megakernels_b200.model_types import DeviceType, ExtraModelConfig


def read_layer(i: int, raw: dict, shape_of) -> LayerSpec:
    m = raw["mixer"]
    if raw["type"] == "general_delta":
        mixer = DeltaRuleSpec(heads=m["heads"], dim=m["dim"], rank=shape_of(f"l{i}.mix.w1")[0])
    elif raw["type"] == "attention":
        mixer = DiffAttentionSpec(
            heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
            window=m["mask"]["size"], keep_first=m["mask"]["keep_first"], diff=m["diff"], kv_from=m.get("kv_from"),
        )
    else:
        raise ValueError(f"layer {i}: unknown mixer type {raw['type']!r}")
    mlp = raw.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return LayerSpec(mixer, None if mlp is None else PolyNormSpec(mlp["ff"]))


def read_config(raw: dict, shape_of) -> HybridConfig:
    """``shape_of(name)`` is a tensor's shape (the low-rank decay's inner size is only there)."""
    return HybridConfig(
        width=raw["width"], vocab_size=raw["vocab"], max_position_embeddings=raw["max_positions"],
        eps=raw["norm"]["eps"], embed_scale=raw["embedding"]["scale"],
        layers=tuple(read_layer(i, layer, shape_of) for i, layer in enumerate(raw["layers"])),
    )


class ToriraxForCausalLM(HybridForCausalLM):
    @classmethod
    def from_pretrained(
        cls,
        model_path: str | Path,
        extra_config: ExtraModelConfig | None = None,
        device: DeviceType = "cuda:0",
        dtype: torch.dtype = torch.bfloat16,
    ) -> "ToriraxForCausalLM":
        from safetensors import safe_open

        path = Path(model_path)
        files = sorted(path.glob("*.safetensors"))
        if not files:
            raise FileNotFoundError(f"no safetensors files under {path}")
        handles = [safe_open(f, framework="pt", device="cpu") for f in files]
        where = {name: h for h in handles for name in h.keys()}
        config = read_config(json.loads((path / "config.json").read_text()),
                             lambda name: where[name].get_slice(name).get_shape())
        return cls.assemble(config, extra_config, device, dtype, lambda name: where[name].get_tensor(name))


# ---- random-weight shapes (layers of a real model's proportions) ---------------------------- #
def preset(width: int, heads: int, dim: int, kv_heads: int, ff: int, vocab: int, groups: int, window: int,
           rank: int, max_positions: int = 32768) -> HybridConfig:
    """``groups`` repetitions of two recurrent layers and one attention layer with a feed-forward;
    every second attention layer reads the keys and values of the one before it."""
    layers: list[LayerSpec] = []
    for g in range(groups):
        layers += [LayerSpec(DeltaRuleSpec(heads=width // 64, dim=64, rank=rank), PolyNormSpec(ff))] * 2
        own = len(layers) - 3  # the attention layer of the previous group
        layers.append(LayerSpec(
            DiffAttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=2 * dim, scale=dim**-0.5, window=window,
                              keep_first=4, diff=0.5, kv_from=own if g % 2 else None),
            PolyNormSpec(ff)))
    return HybridConfig(width=width, vocab_size=vocab, max_position_embeddings=max_positions, eps=1e-5,
                        embed_scale=width**0.5, layers=tuple(layers))


PRESETS = {
    # 1B / 8B class: the widths, feed-forward sizes and vocabulary of the Llama presets
    "torirax-1b": lambda groups=5: preset(2048, 16, 64, 4, 8192, 128256, groups, 1024, 64),
    "torirax-8b": lambda groups=6: preset(4096, 16, 128, 4, 14336, 128256, groups, 2048, 128),
}

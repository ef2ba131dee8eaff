"""Torirax: layer-list decoder of generalized-delta-rule and windowed differential-attention layers.

Reads a checkpoint directory (``config.json``, ``*.safetensors``) into the mechanisms of
``hybrid.py``.  Every size comes from the configuration or a tensor's shape; the decay's
``exp(-1/2)`` and the unit key's ``1e-6`` are constants of the design (defaults of
``DeltaRuleSpec``).
"""

from __future__ import annotations

from megakernels_b200.hybrid import (
    CheckpointForCausalLM,
    DeltaRuleSpec,
    DiffAttentionSpec,
    HybridConfig,
    LayerSpec,
    PolyNormSpec,
)


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


class ToriraxForCausalLM(CheckpointForCausalLM):
    @classmethod
    def read_config(cls, raw: dict, shape_of) -> HybridConfig:
        return HybridConfig(
            width=raw["width"], vocab_size=raw["vocab"], max_position_embeddings=raw["max_positions"],
            eps=raw["norm"]["eps"], embed_scale=raw["embedding"]["scale"],
            layers=tuple(read_layer(i, layer, shape_of) for i, layer in enumerate(raw["layers"])),
        )


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

"""Dumalix: layer-list decoder of chunked rotary attention and latent attention, with a gated
feed-forward beside each mixer and a stretch of layers that runs several times.

Reads a checkpoint directory (``config.json``, ``*.safetensors``) into the mechanisms of
``hybrid.py``.  Every size comes from the configuration or a tensor's shape; the one-plus norms and
the gated unit's 1.702 are constants of the design.
"""

from __future__ import annotations

from megakernels_b200.hybrid import (
    CheckpointForCausalLM,
    ClampedGluSpec,
    HybridConfig,
    LatentAttentionSpec,
    LayerSpec,
    LoopSpec,
    RopeSpec,
    RotaryAttentionSpec,
    YarnSpec,
)


def read_rope(raw: dict) -> RopeSpec:
    y = raw.get("scaling")
    return RopeSpec(raw["dims"], raw["base"], y and YarnSpec(y["factor"], y["original"], y["fast"], y["slow"]))


def read_layer(i: int, raw: dict, canon_taps: int, shape_of) -> LayerSpec:
    m = raw["mixer"]
    if raw["type"] == "attention":
        mixer = RotaryAttentionSpec(
            heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], chunk=m["mask"]["size"],
            rope=read_rope(m["rot"]), conv_taps=m["conv"] or 0 if "conv" in m else shape_of(f"l{i}.mix.q.conv")[1],
        )
    elif raw["type"] == "latent_attention":
        mixer = LatentAttentionSpec(
            heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], rank=m["kv_rank"], scale=m["scale"],
            rope=read_rope(m["rot"]),
        )
    else:
        raise ValueError(f"layer {i}: unknown mixer type {raw['type']!r}")
    mlp = raw.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return LayerSpec(mixer, None if mlp is None else ClampedGluSpec(mlp["ff"], mlp["limit"]), parallel=True, canon_taps=canon_taps)


class DumalixForCausalLM(CheckpointForCausalLM):
    @classmethod
    def read_config(cls, raw: dict, shape_of) -> HybridConfig:
        loop = raw.get("loop")
        return HybridConfig(
            width=raw["width"], vocab_size=raw["vocab"], max_position_embeddings=None, eps=raw["norm"]["eps"], embed_scale=1.0,
            layers=tuple(read_layer(i, layer, raw["canon"]["taps"], shape_of) for i, layer in enumerate(raw["layers"])),
            norm="rms_norm", norm_offset=1.0, learned_positions=False,
            loop=loop and LoopSpec(loop["start"], loop["stop"], loop["times"]),
        )


# ---- random-weight shapes (layers of a real model's proportions) ---------------------------- #
def preset(width: int, heads: int, kv_heads: int, dim: int, latent_heads: int, rank: int, ff: int, vocab: int, layers: int,
           loop: LoopSpec, chunk: int) -> HybridConfig:
    """Latent and chunked attention in turn, every layer with a feed-forward."""
    yarn = YarnSpec(factor=8.0, original=4096, fast=32.0, slow=1.0)
    latent = LatentAttentionSpec(heads=latent_heads, dim=128, rot_dim=64, vdim=128, rank=rank, scale=192**-0.5,
                                 rope=RopeSpec(64, 10000.0, yarn))
    chunked = RotaryAttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim**-0.5, chunk=chunk,
                                  rope=RopeSpec(dim, 500000.0, yarn), conv_taps=4)
    specs = [LayerSpec(chunked if i % 2 else latent, ClampedGluSpec(ff, 7.0), parallel=True, canon_taps=4) for i in range(layers)]
    return HybridConfig(width=width, vocab_size=vocab, max_position_embeddings=None, eps=1e-5, embed_scale=1.0, layers=tuple(specs),
                        norm="rms_norm", norm_offset=1.0, learned_positions=False, loop=loop)


PRESETS = {
    # 1B / 8B class: the widths, feed-forward sizes, vocabulary and layer runs of the Llama presets
    "dumalix-1b": lambda: preset(2048, 32, 8, 64, 16, 512, 8192, 128256, 12, LoopSpec(4, 6, 3), 8192),
    "dumalix-8b": lambda: preset(4096, 32, 8, 128, 32, 512, 14336, 128256, 24, LoopSpec(8, 12, 3), 8192),
}

"""Small Torirax models for the tests: configurations, random tensors, checkpoints, comparisons."""

from __future__ import annotations

import json

import torch

from megakernels_b200.hybrid import tensor_shapes
from megakernels_b200.torirax import ToriraxForCausalLM
from oracle import torirax_ref

F32_TOL, BF16_TOL = 6e-5, 4e-2  # root mean square of the logits' difference over that of the logits


def delta(heads, dim, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": ff and {"kind": "dense", "ff": ff}}


def attention(heads, kv_heads, dim, vdim, size, keep_first, diff=0.4, scale=None, kv_from=None, ff=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, diff=diff, scale=scale or dim**-0.5,
             mask=dict(size=size, keep_first=keep_first))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": ff and {"kind": "dense", "ff": ff}}


def model_config(layers, width=72, vocab=131, max_positions=320, eps=1e-5, scale=3.0):
    return {"architecture": "Torirax", "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers,
            "max_positions": max_positions, "vocab": vocab, "width": width}


# sizes that are no multiples of anything, every branch, unequal masks on one cache
ODD = model_config([
    delta(3, 24, ff=100),
    attention(6, 3, 16, 24, size=11, keep_first=3),
    delta(2, 41),
    attention(6, 3, 16, 24, size=29, keep_first=5, kv_from=1, diff=0.15, ff=52),
    attention(2, 2, 20, 37, size=1, keep_first=0, scale=0.31, ff=33),
    delta(1, 70, ff=17),
    attention(4, 1, 9, 8, size=500, keep_first=1, diff=0.0),
], eps=3e-4)
# sizes of real models' heads, 16-byte rows everywhere
EVEN = model_config([
    delta(4, 64),
    attention(8, 2, 64, 128, size=70, keep_first=4, ff=320),
    delta(2, 128, ff=256),
    attention(8, 2, 64, 128, size=33, keep_first=9, kv_from=1, diff=0.6, ff=192),
    delta(3, 96),
    attention(3, 3, 48, 80, size=17, keep_first=2, ff=512),
], width=192, vocab=260)
WIDE = model_config([delta(1, 256), attention(2, 1, 128, 256, size=90, keep_first=2, ff=1100), delta(2, 160)],
                    width=520, vocab=1031)
# an attention layer first, a width that is no multiple of 4, one kept position, KV heads of their own
RAGGED = model_config([
    attention(3, 3, 12, 40, size=21, keep_first=1, diff=0.7, ff=45),
    attention(3, 3, 12, 40, size=4, keep_first=6, diff=0.25, scale=0.5, kv_from=0),
    delta(5, 12),
    delta(1, 33, ff=66),
], width=71, vocab=97, eps=1e-4, scale=0.8)
MODELS = {"odd": ODD, "even": EVEN, "wide": WIDE, "ragged": RAGGED}


def rank_of(i: int) -> int:
    return (7, 16, 5, 24)[i % 4]


def make_weights(raw, seed=0, qk_gain=1.0):
    """Random bf16 tensors; ``qk_gain`` scales the query and key projections (peaked attention)."""
    gen = torch.Generator().manual_seed(seed)
    layer = lambda name: int(name.split(".")[0][1:])  # noqa: E731
    config = ToriraxForCausalLM.read_config(raw, lambda name: (rank_of(layer(name)), raw["width"]))
    out = {}
    for name, shape in tensor_shapes(config).items():
        w = torch.randn(shape, generator=gen)
        if name in ("embed", "pos"):
            w *= 0.5
        elif len(shape) == 2:
            w *= shape[1] ** -0.5
            if name.split(".")[-1] in ("q", "k") and raw["layers"][layer(name)]["type"] == "attention":
                w *= qk_gain
        elif name.endswith(".act"):
            w = torch.tensor([0.7, -0.4, 0.3, 0.2]) + 0.1 * w
        elif name.endswith((".b", ".lq1", ".lk1", ".lq2", ".lk2")):
            w *= 0.3
        elif name.endswith(".w0"):
            w = 2.0 * w - 1.0
        else:
            w = 1.0 + 0.3 * w  # norms and layer scales
        out[name] = w.to(torch.bfloat16)
    return out


def write_checkpoint(path, raw, weights):
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.contiguous() for k, v in weights.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(raw))
    return path


def tokens_for(raw, n, seed=1):
    return torch.randint(0, raw["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(raw, weights, tokens, **kw):
    return torirax_ref.forward(raw, weights, tokens, **kw)


def rel(got, want) -> float:
    """Worst position: rms of the difference over the rms of all expected logits."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    return float((got - want).pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt())


def load(path, dtype=torch.float32, portion=2048, slots=3, max_len=None, **kw):
    """Generator of a checkpoint through the registry and the dispatch tables."""
    from megakernels_b200.dispatch import make_generator
    from megakernels_b200.model_types import ExtraModelConfig
    from megakernels_b200.registry import load_model

    extra = ExtraModelConfig(max_batch_size=slots, prefill_portion=portion, max_len_override=max_len)
    return make_generator(load_model(path, extra, dtype=dtype), **kw)


def run_cut(gen, tokens, cuts, slot=0, start=0):
    """Feed ``tokens`` in portions of the given sizes (the rest one by one); all logits."""
    out, at = [], start
    cuts = list(cuts)
    while at < len(tokens):
        n = min(cuts.pop(0) if cuts else 1, len(tokens) - at)
        out.append(gen.step(tokens[at : at + n], at, list(range(n)), slot=slot))
        at += n
    return torch.cat(out)

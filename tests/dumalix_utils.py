"""Small Dumalix models for the tests: configurations, random tensors, the plain restatement."""

from __future__ import annotations

import json

import torch

from megakernels_b200.dumalix import DumalixForCausalLM
from megakernels_b200.hybrid import tensor_shapes
from oracle import dumalix_ref
from tests.torirax_utils import BF16_TOL, F32_TOL, load, rel, run_cut, tokens_for, write_checkpoint  # noqa: F401

YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}


def mlp(ff, limit=0.9):
    return {"kind": "dense", "ff": ff, "limit": limit}


def chunked(heads, kv_heads, dim, vdim, size, rot=None, base=300.0, scaling=YARN, conv=4, scale=None, ff=None, limit=0.9):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim**-0.5, conv=conv, mask={"size": size},
             rot={"base": base, "dims": dim // 2 * 2 if rot is None else rot, "scaling": scaling})
    return {"type": "attention", "mixer": m, "mlp": ff and mlp(ff, limit)}


def latent(heads, dim, rot_dim, vdim, rank, base=500.0, scaling=YARN, scale=None, ff=None, limit=0.9):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale or (dim + rot_dim) ** -0.5,
             rot={"base": base, "dims": rot_dim, "scaling": scaling})
    return {"type": "latent_attention", "mixer": m, "mlp": ff and mlp(ff, limit)}


def model_config(layers, width=72, vocab=131, eps=1e-5, taps=4, loop=None):
    raw = {"architecture": "Dumalix", "canon": {"taps": taps}, "norm": {"eps": eps}, "layers": layers, "vocab": vocab, "width": width}
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


# sizes that are no multiples of anything, layers without a feed-forward, the loop first
ODD = model_config([
    chunked(6, 3, 20, 28, size=11, rot=8, conv=3, ff=100),
    latent(3, 12, 6, 10, 20, ff=33, limit=0.4),
    chunked(4, 1, 9, 6, size=29, rot=4, conv=2, scale=0.4),
    latent(5, 7, 2, 13, 19, scale=0.5, scaling=None),
], eps=3e-4, taps=3, loop=(0, 2, 2))
# sizes of real models' heads, 16-byte rows everywhere, a loop in the middle
EVEN = model_config([
    latent(8, 64, 32, 64, 128, ff=320, limit=1.3),
    chunked(8, 2, 64, 64, size=33, ff=192, limit=0.7),
    latent(4, 32, 16, 48, 64, ff=256),
    chunked(4, 4, 32, 96, size=70, rot=16, conv=5, ff=512),
    latent(2, 128, 64, 128, 96),
], width=192, vocab=260, loop=(1, 3, 3))
WIDE = model_config([
    latent(6, 128, 64, 128, 320, ff=1100),
    chunked(5, 1, 128, 256, size=100, base=10000.0, ff=600),
    latent(1, 200, 40, 72, 512),
], width=520, vocab=1031, taps=2)
# the whole model three times, a width that is no multiple of 4, one tap, more taps than the chunk
RAGGED = model_config([
    chunked(3, 3, 12, 40, size=5, conv=7, base=50.0, scaling={"factor": 2.5, "original": 20, "fast": 3.0, "slow": 1.0}),
    latent(7, 5, 4, 3, 11, ff=45),
    chunked(2, 1, 6, 2, size=1, conv=1, ff=21),
], width=71, vocab=97, eps=1e-4, taps=1, loop=(0, 3, 3))
# few wide groups of query heads, a long chunk, one pass of the loop, six taps
GROUPS = model_config([
    chunked(16, 1, 40, 24, size=1000, conv=6, ff=64, limit=0.2),
    latent(12, 24, 8, 16, 40, ff=50),
    chunked(12, 3, 16, 16, size=64, scale=0.7, ff=30),
], width=104, vocab=77, taps=6, loop=(1, 2, 1))
MODELS = {"odd": ODD, "even": EVEN, "wide": WIDE, "ragged": RAGGED, "groups": GROUPS}


def config_of(raw):
    """The framework's configuration, without a checkpoint."""
    def shape_of(name):
        layer = raw["layers"][int(name.split(".")[0][1:])]["mixer"]
        assert name.endswith("mix.q.conv")
        return (layer["heads"] * layer["dim"], layer["conv"])

    return DumalixForCausalLM.read_config(raw, shape_of)


def make_weights(raw, seed=0, qk_gain=1.0):
    """Random bf16 tensors; ``qk_gain`` scales the query and key norms (or projections): peaked attention."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config_of(raw)).items():
        w, last = torch.randn(shape, generator=gen), name.split(".")[-1]
        if name == "embed":
            w *= 0.5
        elif last in ("conv", "canon1"):
            w *= 0.4
            w[:, -1] += 0.6 if last == "conv" else 0.0
        elif len(shape) == 2:
            w *= shape[1] ** -0.5
            if last == "uk":
                w *= qk_gain
        elif last == "sink":
            w = 0.5 + w
        elif name.endswith(("q.norm", "k.norm")):
            w = (1.0 + 0.3 * w) * qk_gain**0.5
        elif last in ("norm1", "norm2") or name == "final.norm":
            w *= 0.3  # stored around zero
        else:
            w = 1.0 + 0.3 * w  # temperatures, the latent's norm
        out[name] = w.to(torch.bfloat16)
    return out


def oracle_logits(raw, weights, tokens, **kw):
    return dumalix_ref.forward(raw, weights, tokens, **kw)


def changed(raw, layer, path, value):
    """A copy of a configuration with one entry of a layer (None: of the model) replaced."""
    raw = json.loads(json.dumps(raw))
    at = raw if layer is None else raw["layers"][layer]
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return raw

"""Model container for decoders whose layers are listed one by one.

Each layer has a mixer - a recurrence or an attention - and an optional feed-forward.  The specs
below describe the mechanisms with their constants as parameters; a design (``torirax.py``) reads
its configuration and checkpoint into them.  As ``llama.py``, this is not a torch forward pass: the
container owns what the kernels' globals are built from (padded, stacked weights; per-slot state).

Weight layout the kernels read: matrices row-major ``[out, in]`` in the model dtype with ``in``
padded with zeros to a multiple of 8; the projections that read the same input are stacked into one
matrix; vectors and biases are float32.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable

import torch
from torch import Tensor

from megakernels_b200.model_types import DeviceType, ExtraModelConfig
from megakernels_b200.state import HybridState


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


# ---- mechanisms -------------------------------------------------------------------------- #
@dataclass(frozen=True)
class DeltaRuleSpec:
    """Generalized delta rule with a low-rank per-channel decay.

    ``S <- diag(w) S - (a u)(u^T S) + k v^T``, ``o = S^T r`` with ``u = k / sqrt(sum k^2 +
    unit_eps)`` and ``w = exp(-decay_scale * sigmoid(w2 tanh(w1 h) + w0))``.
    """

    heads: int
    dim: int
    rank: int
    decay_scale: float = math.exp(-0.5)
    unit_eps: float = 1e-6
    kind = "delta_rule"

    @property
    def inner(self) -> int:
        return self.heads * self.dim

    out_features = inner

    @property
    def in_rows(self) -> int:  # r, k, v, a, g, w1
        return 5 * self.inner + self.rank


@dataclass(frozen=True)
class DiffAttentionSpec:
    """Differential attention (two maps over the same values) in a sliding window that also keeps
    the first ``keep_first`` positions; ``kv_from`` reads another layer's keys and values."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int
    diff: float
    kv_from: int | None = None
    kind = "diff_attention"

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def in_rows(self) -> int:  # q, g, then k, v if the layer has them
        own = 0 if self.kv_from is not None else self.kv_heads * (2 * self.dim + self.vdim)
        return self.heads * (2 * self.dim + self.vdim) + own

    def num_splits(self, sm_count: int, keys_per_split: int = 64, limit: int = 32) -> int:
        """Splits of the visible keys per KV head in a decode step: at most one wave of SMs."""
        most = self.window + self.keep_first
        return max(1, min(-(-most // keys_per_split), sm_count // self.kv_heads or 1, limit))


@dataclass(frozen=True)
class PolyNormSpec:
    """``W_down act(W_up h)`` with ``act(z) = a N(z) + b N(z^2) + c N(z^3) + e``."""

    ff: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: DeltaRuleSpec | DiffAttentionSpec
    mlp: PolyNormSpec | None = None


@dataclass(frozen=True)
class HybridConfig:
    width: int
    vocab_size: int
    max_position_embeddings: int
    eps: float
    embed_scale: float
    layers: tuple[LayerSpec, ...]

    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if m.kind != "diff_attention":
                continue
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} KV heads")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if src is None or src.kind != "diff_attention" or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {m.kv_from} is not an earlier layer with keys of its own")
                if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i}: key/value heads differ from layer {m.kv_from}'s")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


# ---- weights ----------------------------------------------------------------------------- #
@dataclass
class LayerParams:
    """One layer's tensors as the kernels read them."""

    in_w: Tensor
    out_w: Tensor
    norm1: Tensor
    ls1: Tensor
    in_bias: Tensor | None = None
    decay_w2: Tensor | None = None
    decay_w0: Tensor | None = None
    out_norm: Tensor | None = None
    diff_lambda: float = 0.0
    norm2: Tensor | None = None
    ls2: Tensor | None = None
    up_w: Tensor | None = None
    down_w: Tensor | None = None
    act: tuple[float, float, float, float] = (0.0, 0.0, 0.0, 0.0)


def difference_lambda(lq1: Tensor, lk1: Tensor, lq2: Tensor, lk2: Tensor, diff: float) -> float:
    """exp(lq1 . lk1) - exp(lq2 . lk2) + diff: a constant of the layer, folded once at load."""
    a, b = ((x.double() * y.double()).sum() for x, y in ((lq1, lk1), (lq2, lk2)))
    return float(a.exp() - b.exp() + diff)


def pad_matrix(w: Tensor, device, dtype: torch.dtype) -> Tensor:
    rows, cols = w.shape
    out = torch.zeros(rows, pad8(cols), device=device, dtype=dtype)
    out[:, :cols] = w.to(device=device, dtype=dtype)
    return out


class HybridForCausalLM:
    """Weights and per-slot state of a layer-list decoder."""

    setting = "hybrid"  # schedule builder, interpreter and generator (dispatch.py)

    def __init__(
        self,
        config: HybridConfig,
        extra_config: ExtraModelConfig,
        device: DeviceType,
        dtype: torch.dtype,
        embed: Tensor,
        positions: Tensor,
        layers: list[LayerParams],
        final_norm: Tensor,
        head: Tensor,
    ):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"unsupported dtype {dtype}")
        if extra_config.tp_size != 1:
            raise ValueError("layer-list models are not sharded")
        self.config = config
        self.extra_config = extra_config
        self.device = torch.device(device)
        self.dtype = dtype
        self.embed, self.positions = embed, positions
        self.layers, self.final_norm, self.head = layers, final_norm, head
        self.setup_caches()

    def max_len(self) -> int:
        limit = self.config.max_position_embeddings
        return min(self.extra_config.max_len_override or limit, limit)

    def portion(self) -> int:
        """Most tokens one prefill call takes."""
        return min(self.extra_config.prefill_portion, self.max_len())

    def setup_caches(self) -> None:
        self.state = HybridState(self.config, self.extra_config.max_batch_size, self.max_len(), self.portion(),
                                 self.device, self.dtype)

    @property
    def slots(self):
        return self.state.pool

    # ---- construction --------------------------------------------------------------------- #
    @classmethod
    def assemble(
        cls,
        config: HybridConfig,
        extra_config: ExtraModelConfig | None,
        device: DeviceType,
        dtype: torch.dtype,
        get: Callable[[str], Tensor],
    ) -> "HybridForCausalLM":
        """Pad, stack and convert the tensors ``get(name)`` returns.

        Names: ``embed``, ``pos``, ``final.norm``, ``head``; per layer ``l<i>.`` ``norm1``,
        ``ls1``, ``mix.*`` and, with a feed-forward, ``norm2``, ``ls2``, ``mlp.*``.
        """
        device = torch.device(device)
        mat = lambda w: pad_matrix(w, device, dtype)  # noqa: E731
        vec = lambda w: w.to(device=device, dtype=torch.float32).contiguous()  # noqa: E731
        layers = []
        for i, spec in enumerate(config.layers):
            m, p = spec.mixer, f"l{i}."
            mix = lambda *names: [get(f"{p}mix.{n}") for n in names]  # noqa: E731
            if m.kind == "delta_rule":
                bias = torch.zeros(m.in_rows, device=device)
                bias[3 * m.inner : 4 * m.inner] = vec(get(p + "mix.a.b"))
                kw = dict(
                    in_w=mat(torch.cat(mix("r", "k", "v", "a", "g", "w1"))), in_bias=bias,
                    decay_w2=get(p + "mix.w2").to(device=device, dtype=dtype).contiguous(), decay_w0=vec(get(p + "mix.w0")), out_norm=vec(get(p + "mix.norm")),
                )
            else:
                own = ("k", "v") if m.kv_from is None else ()
                bias = torch.zeros(m.in_rows, device=device)
                nq, ng = m.heads * 2 * m.dim, m.heads * m.vdim
                bias[:nq] = vec(get(p + "mix.q.b"))
                if own:
                    bias[nq + ng :] = vec(torch.cat(mix("k.b", "v.b")))
                kw = dict(in_w=mat(torch.cat(mix("q", "g", *own))), in_bias=bias,
                          diff_lambda=difference_lambda(*mix("lq1", "lk1", "lq2", "lk2"), m.diff))
            if kw["in_w"].shape[0] != m.in_rows:
                raise ValueError(f"layer {i}: {kw['in_w'].shape[0]} projection rows, expected {m.in_rows}")
            if spec.mlp is not None:
                kw.update(norm2=vec(get(p + "norm2")), ls2=vec(get(p + "ls2")), up_w=mat(get(p + "mlp.up")),
                          down_w=mat(get(p + "mlp.down")), act=tuple(get(p + "mlp.act").float().tolist()))
            layers.append(LayerParams(out_w=mat(get(p + "mix.o")), norm1=vec(get(p + "norm1")), ls1=vec(get(p + "ls1")), **kw))
        plain = lambda w: w.to(device=device, dtype=dtype).contiguous()  # noqa: E731
        return cls(config, extra_config or ExtraModelConfig(), device, dtype, plain(get("embed")), plain(get("pos")),
                   layers, vec(get("final.norm")), mat(get("head")))

    @classmethod
    def from_random(
        cls,
        config: HybridConfig,
        extra_config: ExtraModelConfig | None = None,
        device: DeviceType = "cuda:0",
        dtype: torch.dtype = torch.bfloat16,
        seed: int = 0,
        draw_on: str = "cpu",
    ) -> "HybridForCausalLM":
        """Seeded random weights: matrices N(0, 1/in), norms and scales around 1, decays spread."""
        where = torch.device(device) if draw_on == "device" else torch.device("cpu")
        gen = torch.Generator(device=where).manual_seed(seed)
        shapes = tensor_shapes(config)

        def get(name: str) -> Tensor:
            shape = shapes[name]
            w = torch.randn(shape, generator=gen, device=where, dtype=torch.float32)
            if len(shape) == 2:
                w *= 0.02 if name in ("embed", "pos") else shape[1] ** -0.5
            elif name.endswith(".act"):
                w = torch.tensor([0.6, 0.3, 0.2, 0.05], device=where) + 0.05 * w
            elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2", ".b")):
                w *= 0.1
            elif not name.endswith(".w0"):
                w = 1.0 + 0.1 * w
            return w.to(torch.bfloat16)  # both dtypes hold the same values

        return cls.assemble(config, extra_config, device, dtype, get)


def tensor_shapes(config: HybridConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor of a model."""
    W = config.width
    out = {"embed": (config.vocab_size, W), "pos": (config.max_position_embeddings, W)}
    for i, spec in enumerate(config.layers):
        m, p = spec.mixer, f"l{i}."
        out[p + "norm1"] = out[p + "ls1"] = (W,)
        if m.kind == "delta_rule":
            out.update({f"{p}mix.{n}": (m.inner, W) for n in "rkvag"})
            out.update({f"{p}mix.{n}": (m.inner,) for n in ("a.b", "w0", "norm")})
            out[p + "mix.w1"], out[p + "mix.w2"] = (m.rank, W), (m.inner, m.rank)
        else:
            sizes = {"q": m.heads * 2 * m.dim, "k": m.kv_heads * 2 * m.dim, "v": m.kv_heads * m.vdim}
            for n in "qkv" if m.kv_from is None else "q":
                out[f"{p}mix.{n}"], out[f"{p}mix.{n}.b"] = (sizes[n], W), (sizes[n],)
            out[p + "mix.g"] = (m.out_features, W)
            out.update({f"{p}mix.{n}": (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        out[p + "mix.o"] = (W, m.out_features)
        if spec.mlp is not None:
            out[p + "norm2"] = out[p + "ls2"] = (W,)
            out[p + "mlp.up"], out[p + "mlp.down"], out[p + "mlp.act"] = (spec.mlp.ff, W), (W, spec.mlp.ff), (4,)
    out["final.norm"], out["head"] = (W,), (config.vocab_size, W)
    return out

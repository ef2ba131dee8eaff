"""Model container for decoders whose layers are listed one by one.

Each layer has a mixer - a recurrence or an attention - and an optional feed-forward, after it or
beside it.  A stretch of layers may run several times with the same weights; a *run* is one use of a
layer, with state of its own.  The specs below describe the mechanisms with their constants as
parameters; a design (``torirax.py``, ``dumalix.py``) reads its configuration and checkpoint into
them.  As ``llama.py``, this is not a torch forward pass: the
container owns what the kernels' globals are built from (padded, stacked weights; per-slot state).

Weight layout the kernels read: matrices row-major ``[out, in]`` in the model dtype with ``in``
padded with zeros to a multiple of 8; the projections that read the same input are stacked into one
matrix; vectors and biases are float32.
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass
from functools import cached_property
from pathlib import Path
from typing import Callable

import torch
from torch import Tensor

from megakernels_b200.model_types import DeviceType, ExtraModelConfig
from megakernels_b200.state import HybridState


DEFAULT_MAX_LEN = 32768  # positions per slot where neither the design nor the caller sets a limit


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

    key_groups = property(lambda self: self.kv_heads)  # attention instructions per split of the keys
    key_elems = property(lambda self: self.kv_heads * (2 * self.dim + self.vdim))  # cached per position


@dataclass(frozen=True)
class YarnSpec:
    """Frequencies of slow pairs divided by ``factor``, of fast pairs kept, a ramp between the pairs
    that turn ``slow`` and ``fast`` times within ``original`` positions; cosine and sine times
    ``0.1 ln(factor) + 1``."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RopeSpec:
    """Rotation of the first ``dims`` elements of a vector, neighbours (2i, 2i + 1) by
    ``position * base^(-2i / dims)``."""

    dims: int
    base: float
    scaling: YarnSpec | None = None

    def frequencies(self) -> tuple[Tensor, float]:
        """float64 ``[dims / 2]`` and the factor of cosine and sine."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = self.base ** (-2.0 * i / self.dims) if self.dims else i
        y = self.scaling
        if y is None or not self.dims:
            return f, 1.0
        pair = lambda turns: self.dims * math.log(y.original / (2 * math.pi * turns)) / (2 * math.log(self.base))  # noqa: E731
        lo, hi = max(math.floor(pair(y.fast)), 0), min(math.ceil(pair(y.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        return f / y.factor * ramp + f * (1 - ramp), 0.1 * math.log(y.factor) + 1

    def table(self, length: int) -> Tensor:
        """float32 ``[length, dims / 2, 2]``: cosine and sine, rounded once from float64."""
        f, factor = self.frequencies()
        angle = torch.arange(length, dtype=torch.float64)[:, None] * f
        return (torch.stack([angle.cos(), angle.sin()], dim=-1) * factor).float()


@dataclass(frozen=True)
class RotaryAttentionSpec:
    """Softmax attention over rotated, normalised queries and keys; a causal convolution over time
    of ``conv_taps`` on the projections; keys of the query's own chunk of ``chunk`` positions; a
    temperature and a sink (a key without a value) per head; ``turn_values``: values are rotated
    over all of ``vdim`` by their position (``rope.base``) and outputs turned back by the query's."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    rope: RopeSpec
    conv_taps: int = 0
    turn_values: bool = True
    kv_from = None
    keep_first = 0
    kind = "attention"

    out_features = property(lambda self: self.heads * self.vdim)
    in_rows = property(lambda self: self.heads * self.dim + self.kv_heads * (self.dim + self.vdim))  # q, k, v
    window = property(lambda self: self.chunk)
    key_groups = property(lambda self: self.kv_heads)
    key_elems = property(lambda self: self.kv_heads * (self.dim + self.vdim))


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Causal attention whose keys and values are expanded from one latent of ``rank`` elements per
    position, next to ``rot_dim`` rotated key elements that all heads share.  The cache holds the
    latent and the rotated part; decode steps attend in latent space (the key expansion is absorbed
    into the query, the value expansion comes after), prefill expands keys and values."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    rope: RopeSpec
    kv_from = None
    keep_first = 0
    window = 1 << 30
    kind = "latent_attention"

    out_features = property(lambda self: self.heads * self.vdim)
    in_rows = property(lambda self: self.heads * (self.dim + self.rot_dim) + self.rank + self.rot_dim)
    row_elems = property(lambda self: ((pad8(self.rank) + pad8(self.rot_dim)) // 8 | 1) * 8)  # of the cache
    key_elems = row_elems

    @property
    def key_groups(self) -> int:
        """Groups of heads that share an attention instruction in a decode step."""
        per = max(p for p in range(1, 9) if self.heads % p == 0)
        return self.heads // per


def key_splits(m, max_len: int, sm_count: int, keys_per_split: int = 64) -> int:
    """Splits of the visible keys per KV head in a decode step: at most one wave of SMs."""
    limit = 64 if m.kind == "latent_attention" else 32  # (what the kernel merges)
    most = min(m.window + m.keep_first, max_len)
    return max(1, min(-(-most // keys_per_split), sm_count // m.key_groups or 1, limit))


@dataclass(frozen=True)
class PolyNormSpec:
    """``W_down act(W_up h)`` with ``act(z) = a N(z) + b N(z^2) + c N(z^3) + e``."""

    ff: int
    kind = "poly_norm"
    up_rows = property(lambda self: self.ff)


@dataclass(frozen=True)
class ClampedGluSpec:
    """``W_down (g sigmoid(alpha g) (u + 1))`` with ``g = min(W_gate h, limit)`` and
    ``u = clamp(W_up h, -limit, limit)``; the kernels read gate and up rows in turn."""

    ff: int
    limit: float
    alpha: float = 1.702
    kind = "clamped_glu"
    up_rows = property(lambda self: 2 * self.ff)


@dataclass(frozen=True)
class LayerSpec:
    """``parallel``: mixer and feed-forward read the same stream and are added to it together.
    ``canon_taps``: a causal convolution over time on what the mixer reads, added to it."""

    mixer: DeltaRuleSpec | DiffAttentionSpec | RotaryAttentionSpec | LatentAttentionSpec
    mlp: PolyNormSpec | ClampedGluSpec | None = None
    parallel: bool = False
    canon_taps: int = 0


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop - 1`` run ``times`` times in a row; before each pass the stream and
    the embedding are projected back to one stream."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class HybridConfig:
    """``norm``: ``layer_norm`` or ``rms_norm``, its stored weights offset by ``norm_offset``."""

    width: int
    vocab_size: int
    max_position_embeddings: int | None
    eps: float
    embed_scale: float
    layers: tuple[LayerSpec, ...]
    norm: str = "layer_norm"
    norm_offset: float = 0.0
    learned_positions: bool = True
    loop: LoopSpec | None = None

    def __post_init__(self):
        if self.loop is not None:
            a, b, n = self.loop.start, self.loop.stop, self.loop.times
            if not (0 <= a < b <= len(self.layers) and n >= 1):
                raise ValueError(f"layers {a}..{b - 1} of {len(self.layers)} run {n} times")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if layer.parallel and layer.mlp is not None and layer.mlp.kind != "clamped_glu":
                raise ValueError(f"layer {i}: a {layer.mlp.kind} feed-forward does not run beside a mixer")
            if getattr(m, "heads", 1) % getattr(m, "kv_heads", 1):
                raise ValueError(f"layer {i}: {m.heads} query heads over {m.kv_heads} KV heads")
            if m.kind != "diff_attention":
                continue
            if m.kv_from is not None and self.loop is not None:
                raise ValueError(f"layer {i}: keys of another layer in a model with a loop")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if src is None or src.kind != "diff_attention" or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {m.kv_from} is not an earlier layer with keys of its own")
                if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i}: key/value heads differ from layer {m.kv_from}'s")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @cached_property
    def runs(self) -> tuple[tuple[int, bool], ...]:
        """(layer, does the run start a pass of the loop) in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return tuple((i, False) for i in range(n))
        a, b = self.loop.start, self.loop.stop
        one = [(i, i == a) for i in range(a, b)]
        return tuple([(i, False) for i in range(a)] + one * self.loop.times + [(i, False) for i in range(b, n)])

    @property
    def run_layers(self) -> list[LayerSpec]:
        return [self.layers[i] for i, _ in self.runs]


# ---- weights ----------------------------------------------------------------------------- #
@dataclass
class LayerParams:
    """One layer's tensors as the kernels read them."""

    in_w: Tensor
    out_w: Tensor
    norm1: Tensor
    ls1: Tensor | None = None
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
    canon_w: Tensor | None = None  # [taps, width]
    canon_gain: Tensor | None = None  # norm1 * (1 + last tap)
    conv_w: Tensor | None = None  # [taps, stacked projection rows]
    q_norm: Tensor | None = None
    k_norm: Tensor | None = None
    temp: Tensor | None = None
    sink: Tensor | None = None
    absorb_w: Tensor | None = None  # [heads * rank, dim]: the key expansion, transposed per head
    expand_w: Tensor | None = None  # [heads * (dim + vdim), rank]: keys of all heads, values of all heads


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
        positions: Tensor | None,
        layers: list[LayerParams],
        final_norm: Tensor,
        head: Tensor,
        enter: Tensor | None = None,
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
        self.layers, self.final_norm, self.head, self.enter = layers, final_norm, head, enter
        self.setup_caches()

    def max_len(self) -> int:
        limit, wanted = self.config.max_position_embeddings, self.extra_config.max_len_override
        if limit is None:  # the design sets none
            return wanted or DEFAULT_MAX_LEN
        return min(wanted or limit, limit)

    def portion(self) -> int:
        """Most tokens one prefill call takes."""
        return min(self.extra_config.prefill_portion, self.max_len())

    def setup_caches(self) -> None:
        self.state = HybridState(self.config, self.extra_config.max_batch_size, self.max_len(), self.portion(),
                                 self.device, self.dtype)
        self._tables: dict[RopeSpec, Tensor] = {}

    def rope_table(self, spec: RopeSpec) -> Tensor:
        """Cosines and sines of every position; one table per kind of rotation."""
        if spec not in self._tables:
            self._tables[spec] = spec.table(self.max_len()).to(self.device)
        return self._tables[spec]

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
        """Pad, stack and convert the tensors ``get(name)`` returns; ``tensor_shapes`` lists the names."""
        device = torch.device(device)
        mat = lambda w: pad_matrix(w, device, dtype)  # noqa: E731
        vec = lambda w: w.to(device=device, dtype=torch.float32).contiguous()  # noqa: E731
        norm = lambda name: vec(get(name)) + config.norm_offset  # noqa: E731
        scaled = config.norm == "layer_norm"  # (designs with layer norms have layer scales)
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
            elif m.kind == "diff_attention":
                own = ("k", "v") if m.kv_from is None else ()
                bias = torch.zeros(m.in_rows, device=device)
                nq, ng = m.heads * 2 * m.dim, m.heads * m.vdim
                bias[:nq] = vec(get(p + "mix.q.b"))
                if own:
                    bias[nq + ng :] = vec(torch.cat(mix("k.b", "v.b")))
                kw = dict(in_w=mat(torch.cat(mix("q", "g", *own))), in_bias=bias,
                          diff_lambda=difference_lambda(*mix("lq1", "lk1", "lq2", "lk2"), m.diff))
            elif m.kind == "attention":
                kw = dict(in_w=mat(torch.cat(mix("q", "k", "v"))), q_norm=vec(get(p + "mix.q.norm")), k_norm=vec(get(p + "mix.k.norm")),
                          temp=vec(get(p + "mix.temp")), sink=vec(get(p + "mix.sink")))
                if m.conv_taps:
                    kw["conv_w"] = vec(torch.cat(mix("q.conv", "k.conv", "v.conv")).T)
            else:
                uk, uv = mix("uk", "uv")
                back = uk.view(m.heads, m.dim, m.rank).transpose(1, 2).reshape(m.heads * m.rank, m.dim)
                kw = dict(in_w=mat(torch.cat(mix("q", "dkv"))), k_norm=vec(get(p + "mix.dkv.norm")), absorb_w=mat(back),
                          expand_w=mat(torch.cat([uk, uv])))
            if kw["in_w"].shape[0] != m.in_rows:
                raise ValueError(f"layer {i}: {kw['in_w'].shape[0]} projection rows, expected {m.in_rows}")
            kw["norm1"] = norm(p + "norm1")
            if spec.canon_taps:
                kw["canon_w"] = vec(get(p + "canon1").T)
                kw["canon_gain"] = (kw["norm1"].double() * (1 + kw["canon_w"][-1].double())).float()
            if scaled:
                kw["ls1"] = vec(get(p + "ls1"))
            if spec.mlp is not None:
                kw.update(norm2=norm(p + "norm2"), down_w=mat(get(p + "mlp.down")))
                if scaled:
                    kw["ls2"] = vec(get(p + "ls2"))
                if spec.mlp.kind == "clamped_glu":
                    kw["up_w"] = mat(torch.stack([get(p + "mlp.gate"), get(p + "mlp.up")], dim=1).flatten(0, 1))
                else:
                    kw.update(up_w=mat(get(p + "mlp.up")), act=tuple(get(p + "mlp.act").float().tolist()))
            layers.append(LayerParams(out_w=mat(get(p + "mix.o")), **kw))
        plain = lambda w: w.to(device=device, dtype=dtype).contiguous()  # noqa: E731
        return cls(config, extra_config or ExtraModelConfig(), device, dtype, plain(get("embed")),
                   plain(get("pos")) if config.learned_positions else None, layers, norm("final.norm"), mat(get("head")),
                   mat(get("loop.in")) if config.loop is not None else None)

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
            elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2", ".b", ".sink")):
                w *= 0.1
            elif name.endswith(("norm1", "norm2", "final.norm")):
                w = 1.0 - config.norm_offset + 0.1 * w
            elif not name.endswith(".w0"):
                w = 1.0 + 0.1 * w
            return w.to(torch.bfloat16)  # both dtypes hold the same values

        return cls.assemble(config, extra_config, device, dtype, get)


class CheckpointForCausalLM(HybridForCausalLM):
    """A design: how its ``config.json`` maps to a ``HybridConfig``."""

    @classmethod
    def read_config(cls, raw: dict, shape_of: Callable[[str], tuple[int, ...]]) -> HybridConfig:
        """``shape_of(name)`` is a tensor's shape (some sizes are only there)."""
        raise NotImplementedError

    @classmethod
    def from_pretrained(
        cls,
        model_path: str | Path,
        extra_config: ExtraModelConfig | None = None,
        device: DeviceType = "cuda:0",
        dtype: torch.dtype = torch.bfloat16,
    ) -> "CheckpointForCausalLM":
        from safetensors import safe_open

        path = Path(model_path)
        files = sorted(path.glob("*.safetensors"))
        if not files:
            raise FileNotFoundError(f"no safetensors files under {path}")
        handles = [safe_open(f, framework="pt", device="cpu") for f in files]
        where = {name: h for h in handles for name in h.keys()}
        config = cls.read_config(json.loads((path / "config.json").read_text()),
                                 lambda name: where[name].get_slice(name).get_shape())
        return cls.assemble(config, extra_config, device, dtype, lambda name: where[name].get_tensor(name))


def tensor_shapes(config: HybridConfig) -> dict[str, tuple[int, ...]]:
    """Name -> shape of every tensor of a model."""
    W = config.width
    scaled = config.norm == "layer_norm"
    out = {"embed": (config.vocab_size, W)}
    if config.learned_positions:
        out["pos"] = (config.max_position_embeddings, W)
    if config.loop is not None:
        out["loop.in"] = (W, 2 * W)
    for i, spec in enumerate(config.layers):
        m, p = spec.mixer, f"l{i}."
        out[p + "norm1"] = (W,)
        if scaled:
            out[p + "ls1"] = (W,)
        if spec.canon_taps:
            out[p + "canon1"] = (W, spec.canon_taps)
        if m.kind == "delta_rule":
            out.update({f"{p}mix.{n}": (m.inner, W) for n in "rkvag"})
            out.update({f"{p}mix.{n}": (m.inner,) for n in ("a.b", "w0", "norm")})
            out[p + "mix.w1"], out[p + "mix.w2"] = (m.rank, W), (m.inner, m.rank)
        elif m.kind == "attention":
            sizes = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
            for n, size in sizes.items():
                out[f"{p}mix.{n}"] = (size, W)
                if m.conv_taps:
                    out[f"{p}mix.{n}.conv"] = (size, m.conv_taps)
            out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (m.dim,)
            out[p + "mix.temp"] = out[p + "mix.sink"] = (m.heads,)
        elif m.kind == "latent_attention":
            out[p + "mix.q"], out[p + "mix.dkv"] = (m.heads * (m.dim + m.rot_dim), W), (m.rank + m.rot_dim, W)
            out[p + "mix.dkv.norm"] = (m.rank,)
            out[p + "mix.uk"], out[p + "mix.uv"] = (m.heads * m.dim, m.rank), (m.heads * m.vdim, m.rank)
        else:
            sizes = {"q": m.heads * 2 * m.dim, "k": m.kv_heads * 2 * m.dim, "v": m.kv_heads * m.vdim}
            for n in "qkv" if m.kv_from is None else "q":
                out[f"{p}mix.{n}"], out[f"{p}mix.{n}.b"] = (sizes[n], W), (sizes[n],)
            out[p + "mix.g"] = (m.out_features, W)
            out.update({f"{p}mix.{n}": (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        out[p + "mix.o"] = (W, m.out_features)
        if spec.mlp is not None:
            ff = spec.mlp.ff
            out[p + "norm2"] = (W,)
            if scaled:
                out[p + "ls2"] = (W,)
            out[p + "mlp.up"], out[p + "mlp.down"] = (ff, W), (W, ff)
            if spec.mlp.kind == "clamped_glu":
                out[p + "mlp.gate"] = (ff, W)
            else:
                out[p + "mlp.act"] = (4,)
    out["final.norm"], out["head"] = (W,), (config.vocab_size, W)
    return out

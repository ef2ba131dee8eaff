"""Plain restatement of the Dumalix decoder, one function per mechanism.

Test infrastructure only: it shares no code with the product path, keeps no cache and computes every
sequence from its first token.  Everything runs in the dtype of the tensors it is given
(the tests use float64).  ``weights`` maps tensor names to tensors, ``config`` is the parsed
``config.json``.
"""

from __future__ import annotations

import math

import torch


# ---- norms, convolution, activations ----------------------------------------------------- #
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_plain(x, weight, eps):
    return rms_unit(x, eps) * weight


def norm_one_plus(x, weight, eps):
    return rms_unit(x, eps) * (1 + weight)


def causal_conv(u, w):
    """u [T, channels], w [channels, taps]; the last tap meets the current token."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[: T - back]
    return y


def clamped_glu(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


# ---- rotation ------------------------------------------------------------------------------ #
def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims, base, scaling):
    """Frequencies and the factor of cos and sin; without ``scaling`` the plain ones and 1."""
    f = plain_frequencies(dims, base)
    if scaling is None:
        return f, 1.0
    place = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))  # noqa: E731
    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / scaling["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, freqs, factor=1.0, sign=1):
    """x [T, ..., n]: neighbours (2i, 2i + 1) turn by sign * position * freqs[i]; the rest passes."""
    T, half = x.shape[0], len(freqs)
    angle = sign * torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    shape = (T,) + (1,) * (x.dim() - 2) + (half,)
    c, s = ((factor * f(angle)).to(x.dtype).view(shape) for f in (torch.cos, torch.sin))
    out = x.clone()
    u, v = x[..., 0 : 2 * half : 2], x[..., 1 : 2 * half : 2]
    out[..., 0 : 2 * half : 2] = u * c - v * s
    out[..., 1 : 2 * half : 2] = v * c + u * s
    return out


# ---- attention ----------------------------------------------------------------------------- #
def chunk_visibility(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def causal_visibility(T):
    return torch.ones(T, T, dtype=torch.bool).tril()


def softmax_with_sink(score, mask, sink=None):
    """Rows of weights; exp(sink) joins the denominator once, without a key or a value."""
    score = score.masked_fill(~mask, float("-inf"))
    top = score.amax(dim=-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(score - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


def attention_mixer(h, get, m, eps):
    T = h.shape[0]
    H, G, D, E, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q, k, v = (causal_conv(h @ get(n).T, get(n + ".conv")) for n in "qkv")
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, E)
    freqs, factor = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q = rotate(norm_plain(q, get("q.norm"), eps), freqs, factor)
    k = rotate(norm_plain(k, get("k.norm"), eps), freqs, factor)
    vfreqs = plain_frequencies(E, rot["base"])
    v = rotate(v, vfreqs)
    mask = chunk_visibility(T, m["mask"]["size"])
    heads = []
    for n in range(H):
        g = n // (H // G)
        score = (q[:, n] @ k[:, g].T) * m["scale"] * get("temp")[n]
        heads.append(softmax_with_sink(score, mask, get("sink")[n]) @ v[:, g])
    o = rotate(torch.stack(heads, dim=1), vfreqs, sign=-1)
    return o.reshape(T, H * E) @ get("o").T


def latent_attention_mixer(h, get, m, eps):
    T = h.shape[0]
    H, D, R, E, rank, rot = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["rot"]
    q = (h @ get("q").T).view(T, H, D + R)
    down = h @ get("dkv").T
    c = norm_plain(down[:, :rank], get("dkv.norm"), eps)
    freqs, factor = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    shared = rotate(down[:, rank:], freqs, factor)
    q_rot = rotate(q[..., D:], freqs, factor)
    k = (c @ get("uk").T).view(T, H, D)
    v = (c @ get("uv").T).view(T, H, E)
    mask = causal_visibility(T)
    heads = []
    for n in range(H):
        score = (q[:, n, :D] @ k[:, n].T + q_rot[:, n] @ shared.T) * m["scale"]
        heads.append(softmax_with_sink(score, mask) @ v[:, n])
    return torch.cat(heads, dim=-1) @ get("o").T


# ---- the model ------------------------------------------------------------------------------- #
def layer_runs(config):
    """(layer, is it the first of a pass) in the order the layers run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    one = [(i, i == start) for i in range(start, stop)]
    return [(i, False) for i in range(start)] + one * loop["times"] + [(i, False) for i in range(stop, n)]


def forward(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the residual stream
    after every layer run."""
    W = lambda name: weights[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x0 = x = W("embed")[tokens]
    for i, enters in layer_runs(config):
        layer, p = config["layers"][i], f"l{i}."
        get = lambda name, p=p: W(f"{p}mix.{name}")  # noqa: E731
        if enters:
            x = torch.cat([x, x0], dim=-1) @ W("loop.in").T
        h = norm_one_plus(x, W(p + "norm1"), eps)
        h = h + causal_conv(h, W(p + "canon1"))
        mixer = {"attention": attention_mixer, "latent_attention": latent_attention_mixer}[layer["type"]]
        y = mixer(h, get, layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            f = norm_one_plus(x, W(p + "norm2"), eps)
            z = clamped_glu(f @ W(p + "mlp.gate").T, f @ W(p + "mlp.up").T, mlp["limit"])
            y = y + z @ W(p + "mlp.down").T
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return norm_one_plus(x, W("final.norm"), eps) @ W("head").T

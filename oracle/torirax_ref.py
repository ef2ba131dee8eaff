"""Plain restatement of the Torirax decoder, one function per mechanism.

Test infrastructure only: it shares no code with the product path, keeps no cache and computes every
sequence from its first token.  Everything runs in the dtype of the tensors it is given
(the tests use float64).  ``weights`` maps tensor names to tensors, ``config`` is the parsed
``config.json``.
"""

from __future__ import annotations

import math

import torch


# ---- norms and activations ------------------------------------------------------------- #
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    """Mean removed, divided by the root of the mean squared deviation, weight, no bias."""
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * weight


def poly_norm(z, coeff, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e with N = division by the vector's root mean square."""
    a, b, c, e = (coeff[i] for i in range(4))
    return a * rms_unit(z, eps) + b * rms_unit(z**2, eps) + c * rms_unit(z**3, eps) + e


# ---- generalized delta rule ------------------------------------------------------------ #
def channel_decay(h, w1, w2, w0):
    """exp(-exp(-1/2) * sigmoid(w2 tanh(w1 h) + w0)): a low-rank, per-channel decay."""
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w1.T) @ w2.T + w0))


def delta_recurrence(r, k, v, w, a, state=None):
    """All inputs [T, heads, dim].  Returns outputs [T, heads, dim] and the last state
    [heads, key channel, value channel]."""
    T, heads, dim = r.shape
    S = torch.zeros(heads, dim, dim, dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros_like(r)
    for t in range(T):
        for n in range(heads):
            u = k[t, n] / torch.sqrt((k[t, n] ** 2).sum() + 1e-6)
            read = u @ S[n]
            S[n] = w[t, n][:, None] * S[n] - torch.outer(a[t, n] * u, read) + torch.outer(k[t, n], v[t, n])
            out[t, n] = S[n].T @ r[t, n]
    return out, S


def delta_mixer(h, get, heads, dim, eps):
    T = h.shape[0]
    shape = (T, heads, dim)
    r, k, v = ((h @ get(n).T).view(shape) for n in "rkv")
    w = channel_decay(h, get("w1"), get("w2"), get("w0")).view(shape)
    a = torch.sigmoid(h @ get("a").T + get("a.b")).view(shape)
    o, _ = delta_recurrence(r, k, v, w, a)
    o = rms_unit(o, eps).reshape(T, heads * dim) * get("norm") * torch.sigmoid(h @ get("g").T)
    return o @ get("o").T


# ---- windowed differential attention ---------------------------------------------------- #
def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def visibility(T, size, keep_first):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def attention_map(q, k, v, scale, mask):
    """One softmax attention: q, k [T, dim], v [T, vdim]."""
    score = (q @ k.T) * scale
    return torch.softmax(score.masked_fill(~mask, float("-inf")), dim=-1) @ v


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def attention_keys_values(h, get):
    return h @ get("k").T + get("k.b"), h @ get("v").T + get("v.b")


def diff_attention_mixer(h, k, v, get, m, eps):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ get("q").T + get("q.b")).view(T, H, 2, D)
    k, v = k.view(T, G, 2, D), v.view(T, G, E)
    mask = visibility(T, m["mask"]["size"], m["mask"]["keep_first"])
    lam = diff_lambda(get("lq1"), get("lk1"), get("lq2"), get("lk2"), m["diff"])
    heads = []
    for n in range(H):
        g = n // (H // G)
        a1, a2 = (attention_map(q[:, n, i], k[:, g, i], v[:, g], m["scale"], mask) for i in (0, 1))
        heads.append(rms_unit(a1 - lam * a2, eps) * (1 - m["diff"]))
    o = torch.cat(heads, dim=-1) * torch.sigmoid(h @ get("g").T)
    return o @ get("o").T


# ---- the model --------------------------------------------------------------------------- #
def forward(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the residual stream
    after every layer."""
    W = lambda name: weights[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    T = tokens.numel()
    x = W("embed")[tokens] * config["embedding"]["scale"] + W("pos")[:T]
    kv = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        get = lambda name, p=p: W(f"{p}mix.{name}")  # noqa: E731
        h = layer_norm(x, W(p + "norm1"), eps)
        if layer["type"] == "general_delta":
            y = delta_mixer(h, get, m["heads"], m["dim"], eps)
        else:
            kv[i] = kv[m["kv_from"]] if m.get("kv_from") is not None else attention_keys_values(h, get)
            y = diff_attention_mixer(h, *kv[i], get, m, eps)
        x = x + y * W(p + "ls1")
        if layer["mlp"] is not None:
            h = layer_norm(x, W(p + "norm2"), eps)
            z = poly_norm(h @ W(p + "mlp.up").T, W(p + "mlp.act"), eps)
            x = x + (z @ W(p + "mlp.down").T) * W(p + "ls2")
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, W("final.norm"), eps) @ W("head").T

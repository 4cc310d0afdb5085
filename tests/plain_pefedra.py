"""The Pefedra design stated plainly: whole sequences, float64, no cache, no batching, one function per mechanism.
It shares no code with the package; the tests compare the engine's logits with :func:`forward`.

Notation: ``x [T, width]`` is the residual stream of one sequence whose tokens stand at positions ``0..T-1``;
``h [T, width]`` the input of a part; ``W[name]`` a tensor of the checkpoint; linear weights are ``[out, in]``; ``p`` the
prefix of a part's tensor names and ``m`` its dictionary of the configuration.
"""

from __future__ import annotations

import math

import torch

DT = torch.float64


def rms(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def biased(h, W, name):
    """W h + b"""
    return h @ W[name].T + W[name + ".b"]


def token_shift(h, share):
    """h_t <- h_t + share * (h_(t-1) - h_t), element by element, with the h_(t-1) of before; zeros stand before the first."""
    before = torch.cat((torch.zeros_like(h[:1]), h[:-1]), dim=0)
    return h + (before - h) * share


def frequencies(dims, base, factor=1.0):
    """f_i = base^(-2i/dims) / factor for i < dims/2."""
    return float(base) ** (-2 * torch.arange(dims // 2, dtype=DT) / dims) / float(factor)


def rotate_halves(x, f, sign=1.0):
    """x [T, heads, D]: lanes i and i + n of the first 2n lanes (n = len(f)) turn by sign * position * f_i."""
    n = f.numel()
    a = sign * torch.arange(x.shape[0], dtype=DT)[:, None] * f[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., :n], x[..., n : 2 * n]
    return torch.cat((u * c - v * s, v * c + u * s, x[..., 2 * n :]), dim=-1)


def rotate(x, rot):
    """Queries or keys by the configuration's ``rot``: dims, base and an optional factor that divides every frequency."""
    if not rot or not rot.get("dims"):
        return x
    return rotate_halves(x, frequencies(rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor", 1.0)))


def in_window(T, size):
    """[T, T] booleans: the query at position i (row) sees the key at position j (column) if 0 <= i - j < size."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size)


def softmax_masked(s, see):
    """s [H, T, T] scores; rows are normalised over the keys that ``see [T, T]`` allows."""
    return torch.softmax(s.masked_fill(~see[None], -math.inf), dim=-1)


def grouped(x, heads):
    """[T, kv_heads, D] -> [T, heads, D]: query head h reads key/value head floor(h / (heads / kv_heads))."""
    return x.repeat_interleave(heads // x.shape[1], dim=1)


def difference_weight(W, p, diff):
    """exp(lq1 . lk1) - exp(lq2 . lk2) + diff"""
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + float(diff)


def differential_attention(h, W, p, m, eps):
    """Two softmax maps a head over the same values; the second is subtracted times one number of the layer, each head's
    result is divided by its root mean square and multiplied by 1 - diff."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = biased(h, W, p + "q").view(T, 2 * H, D)
    k = biased(h, W, p + "k").view(T, 2 * G, D)
    v = grouped(biased(h, W, p + "v").view(T, G, V), H)
    q, k = rotate(q, m.get("rot")).view(T, H, 2, D), rotate(k, m.get("rot")).view(T, G, 2, D)
    see, a = in_window(T, m["mask"]["size"]), []
    for i in range(2):
        s = torch.einsum("ihd,jhd->hij", q[:, :, i], grouped(k[:, :, i], H)) * float(m["scale"])
        a.append(torch.einsum("hij,jhd->ihd", softmax_masked(s, see), v))
    o = rms(a[0] - difference_weight(W, p, m["diff"]) * a[1], eps) * (1.0 - float(m["diff"]))
    return o.reshape(T, H * V) @ W[p + "o"].T


def turned_value_attention(h, W, p, m, eps):
    """Softmax attention with q and k normed over their whole projections, values that are rotated by their own position
    before they are summed and each sum turned back by the query's, and a sigmoid gate per head."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(biased(h, W, p + "q"), eps, W[p + "q.norm"]).view(T, H, D)
    k = rms(biased(h, W, p + "k"), eps, W[p + "k.norm"]).view(T, G, D)
    q, k = rotate(q, m.get("rot")), rotate(k, m.get("rot"))
    f = frequencies(V, m["rot"]["base"])
    v = rotate_halves(biased(h, W, p + "v").view(T, G, V), f)
    s = torch.einsum("ihd,jhd->hij", q, grouped(k, H)) * float(m["scale"])
    o = torch.einsum("hij,jhd->ihd", softmax_masked(s, in_window(T, m["mask"]["size"])), grouped(v, H))
    o = rotate_halves(o, f, sign=-1.0)
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ W[p + "o"].T


def gelu(z):
    """z Phi(z), Phi the normal distribution function"""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def feed_forward(h, W, p):
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


MIXERS = {"attention": differential_attention, "attention_2": turned_value_attention}


def forward(cfg, tensors, tokens, return_layers=False):
    """Logits ``[T, vocab]`` (float64) of one whole sequence; with ``return_layers`` also the stream after every layer."""
    W = {k: v.to(DT) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    seen = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = token_shift(rms(x, eps, W[p + "norm1"]), W[p + "shift"])
        y = MIXERS[layer["type"]](h, W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + feed_forward(rms(x, eps, W[p + "norm2"]), W, p + "mlp.")
        x = x + y
        seen.append(x)
    logits = rms(x, eps, W["final.norm"]) @ W["head"].T
    return (logits, seen) if return_layers else logits

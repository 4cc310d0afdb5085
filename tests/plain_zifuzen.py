"""The Zifuzen design stated plainly: whole sequences, float64, no cache, no batching, one function per mechanism.
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


def layer_norm(x, eps, weight):
    """(x - mean) / sqrt(mean squared deviation + eps) * weight"""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def embedding(W, tokens, scale):
    """Row of the token table times a constant, plus the learned vector of the position."""
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return W["embed"][ids] * float(scale) + W["pos"][: len(ids)]


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def short_conv(u, w):
    """y_t = sum_j w[:, j] * u_(t - taps + 1 + j), zeros before the first token; u [T, C], w [C, taps]."""
    taps = w.shape[1]
    padded = torch.cat((torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u), dim=0)
    return sum(w[:, j] * padded[j : j + u.shape[0]] for j in range(taps))


def unit(x):
    """A vector of length one, nearly: x / sqrt(sum x^2 + 1e-6)."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def spread(x, heads):
    """[T, kv_heads, D] -> [T, heads, D]: head h reads key/value head floor(h / (heads / kv_heads))."""
    return x.repeat_interleave(heads // x.shape[1], dim=1)


def step_sizes(h, W, p):
    """beta [T, heads]"""
    return torch.sigmoid(h @ W[p + "b"].T)


def log_decays(h, W, p):
    """ln g [T, heads], never positive"""
    z = h @ W[p + "a"].T + W[p + "dt_bias"]
    softplus = torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))
    return -torch.exp(W[p + "A_log"]) * softplus


def delta_recurrence(q, k, v, beta, log_g):
    """q, k [T, H, D], v [T, H, V], beta, log_g [T, H] -> o [T, H, V]: per head a matrix S [D, V], zero at the start,
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = S * torch.exp(log_g[t])[:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + torch.einsum("hd,hv->hdv", k[t], u)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def delta_mixer(h, W, p, m, eps):
    """The gated delta rule behind short convolutions, each head's result normed, weighted and gated."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k = unit(q.view(T, G, D)) * D**-0.5, unit(k.view(T, G, D))
    o = delta_recurrence(spread(q, H), spread(k, H), v.view(T, H, V), step_sizes(h, W, p), log_decays(h, W, p))
    o = rms(o, eps, W[p + "norm"]) * silu(h @ W[p + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ W[p + "o"].T


def keys_and_values(h, W, p, m, eps):
    """What an attention layer keeps: normed keys [T, kv_heads, dim] and values [T, kv_heads, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    return rms((h @ W[p + "k"].T).view(T, G, m["dim"]), eps, W[p + "k.norm"]), (h @ W[p + "v"].T).view(T, G, m["vdim"])


def attention(h, W, p, m, eps, kept):
    """Causal softmax attention of normed queries over the keys and values ``kept``, positions entering nowhere."""
    T, H = h.shape[0], m["heads"]
    q = rms((h @ W[p + "q"].T).view(T, H, m["dim"]), eps, W[p + "q.norm"])
    k, v = kept
    s = torch.einsum("ihd,jhd->hij", q, spread(k, H)) * float(m["scale"])
    s = s.masked_fill(torch.ones(T, T).triu(1).bool()[None], -math.inf)
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), spread(v, H))
    return o.reshape(T, -1) @ W[p + "o"].T


def dense(h, W, p):
    z = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return z @ W[p + "down"].T + W[p + "down.b"]


def bounded_expert(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=float(limit))
    u = torch.clamp(h @ W[p + "up"].T, min=-float(limit), max=float(limit))
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def group_scores(c, count):
    """[T, experts] choice scores -> [T, count]: the sum of the two largest of each group of neighbours."""
    g = c.view(c.shape[0], count, -1)
    return g.topk(min(2, g.shape[2]), dim=-1).values.sum(-1)


def router_weights(h, W, p, router):
    """[T, experts] weights, zero for experts that a token does not use."""
    s = torch.sigmoid(h @ W[p + "router"].T)
    c = s + W[p + "correction"]
    groups = router.get("groups")
    if groups:
        best = group_scores(c, groups["count"]).topk(groups["keep"], dim=-1).indices
        open_ = torch.zeros(c.shape[0], groups["count"], dtype=torch.bool).scatter(1, best, True)
        c = c.masked_fill(~open_.repeat_interleave(c.shape[1] // groups["count"], dim=1), -math.inf)
    chosen = torch.zeros_like(s).scatter(1, c.topk(router["top"], dim=-1).indices, 1.0)
    w = s * chosen
    return w / (w.sum(-1, keepdim=True) + 1e-20) * float(router["scale"])


def mixture(h, W, p, mlp):
    w = router_weights(h, W, p, mlp["router"])
    y = sum(w[:, e : e + 1] * bounded_expert(h, W, f"{p}e{e}.", mlp["expert"]["limit"]) for e in range(w.shape[1]))
    if mlp.get("shared"):
        y = y + bounded_expert(h, W, p + "shared.", mlp["shared"]["limit"])
    return y


def soft_cap(logits, cap):
    return cap * torch.tanh(logits / cap)


def forward(cfg, tensors, tokens, return_layers=False):
    """Logits ``[T, vocab]`` (float64) of one whole sequence; with ``return_layers`` also the stream after every layer."""
    W = {k: v.to(DT) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    x = embedding(W, tokens, cfg["embedding"]["scale"])
    seen, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            source = m.get("kv_from")
            if source is None:
                kept[i] = keys_and_values(x, W, p + "mix.", m, eps)
            y = attention(x, W, p + "mix.", m, eps, kept[i if source is None else source])
        else:
            y = delta_mixer(x, W, p + "mix.", m, eps)
        x = x + layer_norm(y, eps, W[p + "norm1"])
        mlp = layer.get("mlp")
        if mlp:
            y = dense(x, W, p + "mlp.") if mlp["kind"] == "dense" else mixture(x, W, p + "mlp.", mlp)
            x = x + layer_norm(y, eps, W[p + "norm2"])
        seen.append(x)
    logits = layer_norm(x, eps, W["final.norm"]) @ W["head"].T
    if cfg.get("logit_softcap"):
        logits = soft_cap(logits, float(cfg["logit_softcap"]))
    return (logits, seen) if return_layers else logits

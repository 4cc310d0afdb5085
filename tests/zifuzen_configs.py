"""Small Zifuzen configurations for the tests, as config.json dictionaries.  They differ from one another in every size and
option: values that are often equal are unequal here (key and value sizes, heads and key/value heads, the two recurrent kinds'
sizes and taps, an expert's and the shared expert's size and limit), and options are exercised at 1 and at their ends (one head, one
tap, one expert a token, one group, every group kept, no shared expert, no groups, no feed-forward, no cap, an embedding scale of
one) as well as away from them."""

from __future__ import annotations


def delta(heads, kv_heads, dim, vdim, conv, kind="delta"):
    return {"type": kind, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv_heads, dim, vdim, scale, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, scale=1.7, groups=None, shared=None):
    """``groups``: (count, keep); ``shared``: (ff, limit)."""
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}
    if shared:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    return mlp


def layer(mixer, mlp=None):
    return {**mixer, "mlp": mlp}


def config(layers, vocab=97, width=40, eps=1e-5, scale=2.5, places=400, cap=12.0):
    d = {"architecture": "Zifuzen", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
         "max_positions": places}
    if cap is not None:
        d["logit_softcap"] = cap
    return d


# odd sizes everywhere: three heads on one q/k head, values wider and narrower than keys, taps from 2 to 5, a layer without a
# feed-forward between two with, attention that reads the pages of a layer three entries in front
ODD = config([
    layer(delta(6, 2, 10, 7, 3), dense(28)),
    layer(attention(6, 2, 10, 6, 0.8), moe(6, 2, 9, 0.9, groups=(3, 2), shared=(11, 0.7))),
    layer(delta(3, 3, 6, 13, 5, "delta_2")),
    layer(attention(3, 3, 12, 14, 0.5), moe(10, 3, 7, 1.3, scale=0.8, groups=(2, 1))),
    layer(attention(4, 2, 10, 6, 0.6, kv_from=1), moe(7, 2, 5, 0.8, shared=(8, 2.0))),
    layer(delta(2, 1, 5, 4, 2), moe(8, 4, 6, 1.1, groups=(4, 3), shared=(4, 0.5))),
], eps=5e-2)
# everything at one or at its end: one head, one tap, one expert a token, groups of one expert, every group kept, one group, an
# embedding scale of one, no cap
ONES = config([
    layer(delta(1, 1, 16, 16, 1), dense(16)),
    layer(attention(1, 1, 16, 16, 0.25), moe(4, 1, 16, 1.0, scale=1.0, groups=(4, 1))),
    layer(delta(2, 2, 1, 1, 4, "delta_2"), moe(2, 2, 16, 0.6, groups=(1, 1), shared=(16, 0.6))),
    layer(attention(2, 1, 16, 16, 0.4, kv_from=1), moe(6, 2, 8, 1.5, groups=(2, 2), shared=(8, 3.0))),
    layer(attention(1, 1, 48, 32, 0.2)),
], vocab=61, width=64, eps=1e-6, scale=1.0, cap=None)
# more heads, states of 32 to 130 rows and up to 80 columns, attention heads of 48 and 112 lanes on the tensor cores
WIDE = config([
    layer(delta(8, 4, 48, 80, 4), moe(16, 4, 32, 1.2, groups=(4, 2), shared=(48, 1.0))),
    layer(attention(12, 4, 48, 80, 0.2), dense(160)),
    layer(delta(4, 2, 130, 36, 4, "delta_2"), moe(12, 3, 24, 0.9, groups=(3, 1))),
    layer(attention(8, 4, 112, 16, 0.15), dense(72)),
    layer(attention(4, 4, 112, 16, 0.1, kv_from=3), moe(9, 2, 40, 1.4, shared=(16, 0.8))),
    layer(delta(2, 2, 96, 64, 3), dense(100)),
], vocab=128, width=128, eps=1e-5, scale=4.0, cap=20.0, places=600)
# the sizes that long portions of prompts take to the tcgen05 attention kernel, and states in which a head's columns fill CTAs of
# 64 and of 16
TALL = config([
    layer(delta(4, 2, 64, 128, 4), dense(96)),
    layer(attention(4, 2, 64, 64, 0.3), moe(8, 2, 32, 1.0, groups=(2, 1), shared=(32, 1.0))),
    layer(delta(2, 2, 128, 64, 4, "delta_2"), dense(64)),
    layer(attention(2, 1, 128, 128, 0.2)),
    layer(attention(4, 2, 64, 64, 0.2, kv_from=1), moe(8, 2, 16, 1.2, groups=(4, 2))),
    layer(delta(1, 1, 200, 24, 2), dense(48)),
], vocab=80, width=80, eps=1e-5, scale=3.0, places=700)

ALL = {"odd": ODD, "ones": ONES, "wide": WIDE}

"""Small Pefedra configurations for the tests, as config.json dictionaries.  They differ from one another in every size and
option: values that are often equal are unequal here (key and value sizes, heads and key/value heads, rotated lanes and the head
size, the windows of neighbouring layers), and options are exercised at 1 and at their ends (one head, a window of one, no rotated
lanes, no frequency scaling and a factor below one, a difference weight of zero, no feed-forward, an embedding scale of one) as
well as away from them."""

from __future__ import annotations


def _rot(dims, base, factor):
    rot = {"base": base, "dims": dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return rot


def differential(heads, kv_heads, dim, vdim, scale, size, diff=0.4, dims=None, base=10000.0, factor=None):
    """The ``attention`` mixer: two score maps a head over the same values."""
    return {"type": "attention", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}, "diff": diff,
        "rot": _rot(dim if dims is None else dims, base, factor)}}


def turned(heads, kv_heads, dim, vdim, scale, size, dims=None, base=10000.0):
    """The ``attention_2`` mixer: norms over whole projections, rotated values, a gate per head."""
    return {"type": "attention_2", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
        "rot": _rot(dim if dims is None else dims, base, None)}}


def layer(mixer, ff=None):
    return {**mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=97, width=40, eps=1e-5, scale=2.5):
    return {"architecture": "Pefedra", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}}


# odd sizes everywhere: three query heads on one key/value head, fewer rotated lanes than the head has, values wider and narrower
# than keys, an odd value size, windows that end inside pages, a layer without a feed-forward between two with
ODD = config([
    layer(differential(3, 1, 10, 14, 0.5, 7, diff=0.3, dims=4, base=100.0, factor=3.0), 28),
    layer(turned(4, 2, 6, 10, 0.6, 9, dims=2, base=40.0)),
    layer(turned(3, 3, 12, 6, 0.4, 13), 17),
    layer(differential(2, 2, 6, 5, 0.5, 11, diff=0.7, dims=6), 36),
])
# everything at one or at its end: one head, windows of one, no rotated lanes, a factor of one and below one, a difference
# constant of zero, an embedding scale of one, sizes that the tensor-core kernels take
ONES = config([
    layer(differential(1, 1, 16, 16, 0.25, 1, diff=0.0, dims=0), 16),
    layer(turned(1, 1, 16, 16, 0.25, 1, dims=0)),
    layer(turned(4, 1, 16, 32, 0.3, 20, dims=8), 48),
    layer(differential(4, 1, 16, 48, 0.3, 12, diff=0.9, factor=1.0)),
    layer(differential(2, 2, 32, 16, 0.2, 30, diff=0.2, dims=16, factor=0.5), 64),
], vocab=61, width=64, eps=1e-6, scale=1.0)
# more heads, wide value rows, windows longer than the requests, head sizes of 48 and 80 lanes on the tensor cores
WIDE = config([
    layer(turned(12, 4, 48, 80, 0.15, 25, dims=20, base=500.0), 160),
    layer(differential(6, 2, 80, 128, 0.12, 500, diff=0.5, dims=48, base=700.0, factor=4.0), 72),
    layer(differential(5, 5, 16, 144, 0.2, 17, diff=0.8), 100),
    layer(turned(2, 2, 112, 16, 0.1, 500), 96),
], vocab=128, width=128, eps=1e-5, scale=4.0)

# the sizes that long portions of prompts take to the tcgen05 kernel, with windows shorter and longer than its tiles
TALL = config([
    layer(turned(4, 2, 64, 64, 0.12, 90, dims=48), 80),
    layer(differential(2, 1, 64, 128, 0.15, 140, diff=0.4, factor=2.0), 96),
    layer(differential(3, 3, 64, 64, 0.12, 33, diff=0.6, dims=24)),
    layer(turned(2, 1, 128, 128, 0.1, 600), 64),
    layer(turned(2, 1, 64, 128, 0.12, 65), 112),
], vocab=80, width=80, eps=1e-5, scale=3.0)

ALL = {"odd": ODD, "ones": ONES, "wide": WIDE}

"""The Pefedra design in the engine against the plain implementation (tests/plain_pefedra.py).

Every test makes its own small configuration and random weights.  The engine runs the requests in some way of cutting the work
(whole, token by token, in portions down to two tokens, in mixed batches over a pool so small that pages and state slots are used
again) and the logits at every position are compared with the plain implementation's, which knows no cache.  On the GPU the
engine's kernels run, in true 32-bit and in bfloat16; without one the same host logic runs over the plain operations.
"""

from __future__ import annotations

import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import pefedra_configs as configs
import plain_ops
import plain_pefedra
from test_kafepel import Driver, engine, make_model, tokens_for  # noqa: F401  (the same harness; ``engine`` is a fixture)
from test_nudodra import check

WHERE = ["plain", pytest.param("cuda-float32", marks=pytest.mark.gpu), pytest.param("cuda-bfloat16", marks=pytest.mark.gpu)]
ROOT = Path(__file__).resolve().parent.parent


def expected_of(cfg, tensors, requests):
    return {r: plain_pefedra.forward(cfg, tensors, t) for r, t in requests.items()}


def _loud(tensors):
    """Weights that random draws would leave near nothing, or near one another, made so that leaving them out shows: biases, the
    token shift (shares on both sides of nothing and all), the vectors behind the difference's weight, the whole-projection norms."""
    g = torch.Generator().manual_seed(99)
    for name, t in tensors.items():
        if name.endswith(".shift"):
            tensors[name] = (torch.rand(t.shape, generator=g) * 1.4 - 0.2).to(t.dtype)
        elif name.endswith(".b"):
            tensors[name] = (torch.randn(t.shape, generator=g) * 0.4).to(t.dtype)
        elif name.rsplit(".", 1)[-1] in ("lq1", "lk1", "lq2", "lk2"):
            tensors[name] = (torch.randn(t.shape, generator=g) * 0.7 * t.numel() ** -0.25).to(t.dtype)
        elif name.endswith(("q.norm", "k.norm")):
            tensors[name] = (1.0 + torch.randn(t.shape, generator=g) * 0.3).to(t.dtype)
        elif name.endswith(".mix.g"):
            tensors[name] = (torch.randn(t.shape, generator=g) * 2.0 * t.shape[1] ** -0.5).to(t.dtype)


# --------------------------------------------------------------------------------------------- the plain statement
def test_plain_mechanisms_one_by_one():
    """The oracle's own parts against what they are by definition, on inputs where the answer is known."""
    f64 = torch.float64
    x = torch.randn(7, 2, 6, dtype=f64)
    y = plain_pefedra.rotate(x, {"dims": 4, "base": 10.0})
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])  # position 0 and the lanes behind the rotated ones
    three = torch.tensor(3.0, dtype=f64)  # the first pair's frequency is 1
    assert torch.allclose(y[3, 0, 0], x[3, 0, 0] * torch.cos(three) - x[3, 0, 2] * torch.sin(three))
    assert torch.allclose(y[3, 0, 2], x[3, 0, 2] * torch.cos(three) + x[3, 0, 0] * torch.sin(three))
    slow = torch.tensor(5 * 10.0 ** -0.5 / 4.0, dtype=f64)  # the second pair, with every frequency divided by four
    y = plain_pefedra.rotate(x, {"dims": 4, "base": 10.0, "scaling": {"factor": 4.0}})
    assert torch.allclose(y[5, 1, 1], x[5, 1, 1] * torch.cos(slow) - x[5, 1, 3] * torch.sin(slow))
    f = plain_pefedra.frequencies(6, 10.0)
    assert torch.allclose(plain_pefedra.rotate_halves(plain_pefedra.rotate_halves(x, f), f, sign=-1.0), x)  # turned and turned back
    w = plain_pefedra.in_window(9, 3)
    assert w[8].tolist() == [False] * 6 + [True] * 3 and w[1].tolist() == [True, True] + [False] * 7
    h = torch.tensor([[1.0, 2.0], [10.0, 20.0], [100.0, 200.0]], dtype=f64)
    y = plain_pefedra.token_shift(h, torch.tensor([0.25, 1.0], dtype=f64))
    assert y.tolist() == [[0.75, 0.0], [7.75, 2.0], [77.5, 20.0]]
    z = torch.tensor([0.0, 1.0, -1.0], dtype=f64)
    assert torch.allclose(plain_pefedra.gelu(z), torch.tensor([0.0, 0.8413447460685429, -0.15865525393145707], dtype=f64))
    ones = torch.ones(3, dtype=f64)
    W = {"lq1": ones, "lk1": ones * 0.5, "lq2": ones, "lk2": ones * 0.25}
    assert torch.allclose(plain_pefedra.difference_weight(W, "", 0.6), torch.exp(torch.tensor(1.5, dtype=f64)) - torch.exp(torch.tensor(0.75, dtype=f64)) + 0.6)
    # two equal maps, weight 1/2: half the values' mean, normed to the sign of a single lane, times 1 - diff
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "mask": {"size": 2}, "scale": 1.0, "diff": 0.5, "rot": {"dims": 0, "base": 1.0}}
    zero = torch.zeros(2, dtype=f64)
    W = {"q": torch.zeros(4, 1, dtype=f64), "q.b": torch.zeros(4, dtype=f64), "k": torch.zeros(4, 1, dtype=f64), "k.b": torch.zeros(4, dtype=f64),
         "v": -torch.ones(1, 1, dtype=f64), "v.b": torch.zeros(1, dtype=f64), "o": torch.ones(1, 1, dtype=f64), "lq1": zero, "lk1": zero, "lq2": zero, "lk2": zero}
    out = plain_pefedra.differential_attention(torch.tensor([[1.0], [3.0]], dtype=f64), W, "", m, 0.0)
    assert torch.allclose(out, torch.full((2, 1), -0.5, dtype=f64))
    # rotated values, two keys of equal score: the older value arrives turned back by the one position between them
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 2, "mask": {"size": 2}, "scale": 1.0, "rot": {"dims": 0, "base": 7.0}}
    W = {"q": torch.zeros(1, 2, dtype=f64), "q.b": torch.zeros(1, dtype=f64), "q.norm": torch.ones(1, dtype=f64), "k": torch.zeros(1, 2, dtype=f64),
         "k.b": torch.zeros(1, dtype=f64), "k.norm": torch.ones(1, dtype=f64), "v": torch.eye(2, dtype=f64), "v.b": torch.zeros(2, dtype=f64),
         "g": torch.zeros(1, 2, dtype=f64), "o": 4.0 * torch.eye(2, dtype=f64)}
    out = plain_pefedra.turned_value_attention(torch.tensor([[1.0, 0.0], [0.0, 0.0]], dtype=f64), W, "", m, 1e-5)
    one = torch.tensor(1.0, dtype=f64)
    assert torch.allclose(out[0], torch.tensor([2.0, 0.0], dtype=f64)) and torch.allclose(out[1], torch.stack((torch.cos(one), -torch.sin(one))))


# --------------------------------------------------------------------------------------------- mechanisms alone
ALONE = {
    "differential": configs.config([configs.layer(configs.differential(6, 2, 10, 6, 0.6, 30, dims=6, base=50.0, factor=2.0))], width=32),
    "differential_16": configs.config([configs.layer(configs.differential(4, 2, 32, 48, 0.3, 12, dims=8))], width=32),
    "differential_odd_values": configs.config([configs.layer(configs.differential(2, 1, 6, 7, 0.6, 9))], width=30),
    "turned_values": configs.config([configs.layer(configs.turned(6, 2, 10, 6, 0.7, 30, dims=4))], width=32),
    "turned_values_48": configs.config([configs.layer(configs.turned(8, 2, 16, 48, 0.4, 9))], width=32),
    "turned_values_narrow": configs.config([configs.layer(configs.turned(3, 3, 48, 16, 0.3, 20, dims=16, base=9.0))], width=64),
    "feed_forward": configs.config([configs.layer(configs.differential(1, 1, 4, 4, 0.5, 1), 40)], width=32),
    "feed_forward_64": configs.config([configs.layer(configs.turned(1, 1, 16, 64, 0.5, 1), 128)], width=64),
    "window_of_one": configs.config([configs.layer(configs.turned(2, 1, 16, 32, 0.5, 1)), configs.layer(configs.differential(2, 1, 16, 32, 0.5, 1))], width=48),
}


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone_whole_and_token_by_token(name, where, engine):
    """One or two layers in which one mechanism carries the weight: the whole prompt in one step, and the same tokens one by one
    through the pages and the state."""
    engine(where)
    cfg = ALONE[name]
    model, tensors, dtype = make_model(cfg, 11, where, std=0.2, change=_loud)
    reqs = tokens_for(cfg["vocab"], [37], 5)
    exp = expected_of(cfg, tensors, reqs)
    d = Driver(model, num_pages=24)
    d.run([("r0", reqs["r0"])], end=["r0"])
    check(d.got, exp, dtype, "whole")
    d.got.clear()
    for i, t in enumerate(reqs["r0"]):
        d.run([("r0", [t])], end=["r0"] if i == len(reqs["r0"]) - 1 else [])
    check(d.got, exp, dtype, "token by token")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_residual_stream_after_every_layer(name, where, engine):
    engine(where)
    cfg = configs.ALL[name]
    model, tensors, dtype = make_model(cfg, 3, where, change=_loud)
    tokens = tokens_for(cfg["vocab"], [19], 2)["r0"]
    _, layers = plain_pefedra.forward(cfg, tensors, tokens, return_layers=True)
    seen = []
    model.layer_probe = lambda i, x: seen.append(x.float().cpu().clone())
    Driver(model, num_pages=16).run([("r0", tokens)], end=["r0"])
    assert len(seen) == len(layers) == len(cfg["layers"])
    tol = 1e-4 if dtype == "float32" else 6e-2
    for i, x in enumerate(seen):
        scale = float(layers[i].abs().max())
        assert float((x - layers[i].float()).abs().max()) <= tol * scale, f"the stream differs after layer {i}"


# --------------------------------------------------------------------------------------------- ways of cutting
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_ways_of_cutting(name, where, engine):
    """Whole prompts; a prompt then its last tokens one by one; portions of changing size down to two tokens and one; the first
    tokens of a sequence alone."""
    engine(where)
    cfg = configs.ALL[name]
    model, tensors, dtype = make_model(cfg, 7, where, change=_loud)
    reqs = tokens_for(cfg["vocab"], [1, 2, 45, 83], 9)
    exp = expected_of(cfg, tensors, reqs)
    d = Driver(model, num_pages=24)
    for r, t in reqs.items():
        d.run([(r, t)], end=[r])
    check(d.got, exp, dtype, "whole")
    d.got.clear()
    t = reqs["r3"]
    d.run([("r3", t[:40])])
    for i in range(40, len(t)):
        d.run([("r3", [t[i]])], end=["r3"] if i == len(t) - 1 else [])
    check(d.got, exp, dtype, "decode")
    d.got.clear()
    for r in ("r2", "r3"):
        t, i, k = reqs[r], 0, 0
        sizes = (1, 2, 7, 2, 16, 3, 5, 2, 1, 9)
        while i < len(t):
            n = min(sizes[k % len(sizes)], len(t) - i)
            d.run([(r, t[i : i + n])], end=[r] if i + n == len(t) else [])
            i, k = i + n, k + 1
    check(d.got, exp, dtype, "portions")


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_mixed_batches_with_pages_and_slots_used_again(name, where, engine):
    """Up to four unequal requests a step, portions beside single tokens, over a pool of few pages and four state slots: every
    request's logits equal those of the request alone, also on pages and slots that others gave back (a slot's row of the token
    shift must start at zero again; pages that a window has passed go back early)."""
    engine(where)
    cfg = configs.ALL[name]
    model, tensors, dtype = make_model(cfg, 13, where, change=_loud)
    base = tokens_for(cfg["vocab"], [50, 9, 31, 64, 3, 40], 21)
    exp = expected_of(cfg, tensors, base)
    reqs = {**base, **{r + "#2": t for r, t in base.items()}}  # each once more, on used pages and slots
    prefill = {r: max(1, len(t) - 6) for r, t in reqs.items()}
    d = Driver(model, num_pages=52, page_size=4, max_requests=4)
    waiting, live = list(reqs), {}
    while waiting or live:
        if waiting and len(live) < 4:
            live[waiting.pop(0)] = 0
        entries, end = [], []
        for r, fed in list(live.items()):
            t = reqs[r]
            n = min(7, prefill[r] - fed) if fed < prefill[r] else 1
            n = min(n, len(t) - fed)
            entries.append((r, t[fed : fed + n]))
            live[r] = fed + n
            if live[r] == len(t):
                end.append(r)
                del live[r]
        d.run(entries, end=end)
    assert len({k[0] for k in d.got}) == len(reqs)
    check(d.got, exp, dtype, "mixed")
    assert d.cache.slots.num_used == 0 and all(g.allocator.num_used == 0 for g in d.cache.groups)


@pytest.mark.parametrize("where", WHERE)
def test_a_request_left_out_of_steps_goes_on_where_it_was(where, engine):
    """A request that sits out steps while another takes a slot, steps and ends: its shift row and pages are as it left them."""
    engine(where)
    cfg = configs.ODD
    model, tensors, dtype = make_model(cfg, 19, where, change=_loud)
    reqs = tokens_for(cfg["vocab"], [30, 22], 31)
    exp = expected_of(cfg, tensors, reqs)
    d = Driver(model, num_pages=24, max_requests=2)
    a, b = reqs["r0"], reqs["r1"]
    d.run([("r0", a[:11])])
    d.run([("r1", b[:20])])
    d.run([("r1", b[20:21])])
    d.run([("r1", b[21:])], end=["r1"])
    d.run([("r0", a[11:13])])
    for i in range(13, 30):
        d.run([("r0", [a[i]])], end=["r0"] if i == 29 else [])
    check(d.got, exp, dtype, "left out and taken up again")


@pytest.mark.parametrize("where", WHERE)
def test_long_decoding_over_pages_and_windows(where, engine):
    """A short prompt, then many tokens one by one: pages fill one after the other and go back behind windows, the shift's row
    moves on at every step, and every window's edge is passed token by token."""
    engine(where)
    cfg = configs.ODD
    model, tensors, dtype = make_model(cfg, 17, where, change=_loud)
    t = tokens_for(cfg["vocab"], [150], 4)["r0"]
    exp = expected_of(cfg, tensors, {"r0": t})
    d = Driver(model, num_pages=40, page_size=4)
    d.run([("r0", t[:3])])
    for i in range(3, len(t)):
        d.run([("r0", [t[i]])], end=["r0"] if i == len(t) - 1 else [])
    check(d.got, exp, dtype, "long decoding")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg", [configs.WIDE, configs.TALL], ids=["wide", "tall"])
def test_long_portions(dtype, cfg, engine):
    """Prompts of some hundred tokens, whole and in two long portions beside a decoding request; then single tokens over a context
    long enough to be shared out over several CTAs."""
    where = f"cuda-{dtype}"
    engine(where)
    model, tensors, dtype = make_model(cfg, 23, where, change=_loud)
    reqs = tokens_for(cfg["vocab"], [330, 40], 6)
    exp = expected_of(cfg, tensors, reqs)
    d = Driver(model, num_pages=100, page_size=8)
    d.run([("r0", reqs["r0"])], end=["r0"])
    check(d.got, exp, dtype, "whole")
    d.got.clear()
    d.run([("r1", reqs["r1"][:39])])
    d.run([("r0", reqs["r0"][:150]), ("r1", reqs["r1"][39:])], end=["r1"])
    d.run([("r0", reqs["r0"][150:320])])
    for i in range(320, 330):
        d.run([("r0", [reqs["r0"][i]])], end=["r0"] if i == 329 else [])
    check(d.got, exp, dtype, "two long portions, then single tokens")


# --------------------------------------------------------------------------------------------- faults that random weights would hide
SHARP = {
    # windows of 9 and of 33 with pages of 4, so that the edge falls inside pages and on their borders in turn
    "differential": configs.config([configs.layer(configs.differential(2, 1, 16, 16, 1.0, 9, diff=0.5, dims=4, base=100.0))], width=32),
    "differential_general": configs.config([configs.layer(configs.differential(2, 2, 10, 6, 1.0, 33, diff=0.2, factor=2.0))], width=32),
    "turned": configs.config([configs.layer(configs.turned(2, 1, 16, 16, 4.0, 9, dims=4, base=100.0))], width=32),
    "turned_general": configs.config([configs.layer(configs.turned(2, 2, 10, 6, 4.0, 33))], width=32),
}


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", sorted(SHARP))
def test_keys_at_the_edges_decide(name, where, engine):
    """One attention layer whose scores are sharp: every position leans on one or two keys, which over some hundred positions are
    in turn the key just inside the window, keys at page borders and the query's own; the plain statement with a window that is one
    key wider or narrower differs from the right one by far more than the tolerance.  Prompt in portions that end inside pages,
    then single tokens."""
    engine(where)
    cfg = SHARP[name]
    model, tensors, dtype = make_model(cfg, 29, where, std=0.3, change=_loud)
    t = tokens_for(cfg["vocab"], [260], 12)["r0"]
    exp = expected_of(cfg, tensors, {"r0": t})
    for change in (-1, 1):  # the window matters in this model: one key more or fewer moves the logits visibly
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["mask"]["size"] += change
        assert float((plain_pefedra.forward(other, tensors, t) - exp["r0"]).abs().max()) > 0.1
    d = Driver(model, num_pages=70, page_size=4)
    i = 0
    for n in (3, 126, 2, 70, 39):
        d.run([("r0", t[i : i + n])])
        i += n
    for j in range(i, len(t)):
        d.run([("r0", [t[j]])], end=["r0"] if j == len(t) - 1 else [])
    check(d.got, exp, dtype, "sharp scores")


@pytest.mark.parametrize("what", ["shift", "lambda", "diff", "bias", "norm", "value turn", "gate", "factor", "embedding scale", "feed-forward input"])
def test_every_mechanism_shows_in_the_plain_statement(what, monkeypatch):
    """The weights of these tests are such that leaving a mechanism out moves the plain statement's logits by far more than any
    tolerance here: what the engine is compared with would not forgive it."""
    cfg = json.loads(json.dumps(configs.ODD))
    model, tensors, _ = make_model(cfg, 7, "plain", change=_loud)
    t = tokens_for(cfg["vocab"], [45], 9)["r0"]
    right = plain_pefedra.forward(cfg, tensors, t)
    tensors = dict(tensors)
    P = plain_pefedra
    if what == "shift":
        monkeypatch.setattr(P, "token_shift", lambda h, s: h)
    elif what == "lambda":
        monkeypatch.setattr(P, "difference_weight", lambda W, p, diff: float(diff))
    elif what == "diff":
        cfg["layers"][0]["mixer"]["diff"] = 0.0
    elif what == "bias":
        tensors = {n: (torch.zeros_like(x) if n.endswith("mix.v.b") else x) for n, x in tensors.items()}
    elif what == "norm":
        tensors = {n: (torch.ones_like(x) if n.endswith("q.norm") else x) for n, x in tensors.items()}
    elif what == "value turn":
        turn = P.rotate_halves
        monkeypatch.setattr(P, "rotate_halves", lambda x, f, sign=1.0: x if sign < 0 else turn(x, f))
    elif what == "gate":
        tensors = {n: (torch.zeros_like(x) if n.endswith("mix.g") else x) for n, x in tensors.items()}
    elif what == "factor":
        del cfg["layers"][0]["mixer"]["rot"]["scaling"]
    elif what == "embedding scale":
        cfg["embedding"]["scale"] = 1.0
    else:  # the feed-forward reads the shifted rows instead of a norm of its own
        tensors = {n: (tensors[n[:-1] + "1"] if n.endswith("norm2") else x) for n, x in tensors.items()}
    wrong = P.forward(cfg, tensors, t)
    d = wrong - right
    assert float((d - d.mean(-1, keepdim=True)).pow(2).mean().sqrt() / right.pow(2).mean().sqrt()) > 0.05


# --------------------------------------------------------------------------------------------- configuration and plan
def test_configuration_round_trip_and_errors():
    from llmserve_triton_kernels_b200.config import ConfigError, PefedraConfig, architecture_of

    for cfg in configs.ALL.values():
        typed = architecture_of(cfg).config_class.from_dict(cfg)
        assert isinstance(typed, PefedraConfig) and typed.to_dict() == cfg
        assert PefedraConfig.from_dict(typed.to_dict()) == typed
    for path, value, match in (
        (("layers", 0, "mixer", "diff"), None, "diff"), (("layers", 1, "mixer", "vdim"), 7, "even"), (("layers", 0, "mixer", "kv_heads"), 2, "multiple"),
        (("layers", 2, "type"), "retention", "retention"), (("layers", 0, "mlp", "kind"), "moe", "moe"), (("layers", 1, "mixer", "rot", "dims"), 8, "dims"),
        (("layers", 1, "mixer", "mask", "size"), 0, "mask.size"), (("width",), None, "width"),
    ):
        bad = json.loads(json.dumps(configs.ODD))
        at = bad
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        with pytest.raises(ConfigError, match=match):
            PefedraConfig.from_dict(bad)


def test_plan_names_every_tensor_of_the_design_and_what_layers_keep():
    model, _, _ = make_model(configs.ODD, 1, "plain")
    specs = model.tensor_specs()
    shapes = {
        "embed": (97, 40), "head": (97, 40), "final.norm": (40,), "l0.norm1": (40,), "l0.norm2": (40,), "l0.shift": (40,), "l0.mix.q": (60, 40),
        "l0.mix.q.b": (60,), "l0.mix.k": (20, 40), "l0.mix.v": (14, 40), "l0.mix.v.b": (14,), "l0.mix.lq1": (10,), "l0.mix.lk2": (10,), "l0.mix.o": (40, 42),
        "l0.mlp.up": (28, 40), "l0.mlp.down": (40, 28), "l1.shift": (40,), "l1.mix.q": (24, 40), "l1.mix.q.norm": (24,), "l1.mix.k.norm": (12,),
        "l1.mix.g": (4, 40), "l1.mix.o": (40, 40), "l3.mix.o": (40, 10),
    }
    for name, shape in shapes.items():
        assert specs[name].shape == shape, name
    for name in ("l1.norm2", "l1.mlp.up", "l0.mix.q.norm", "l0.mix.g", "l1.mix.lq1"):
        assert name not in specs, name
    kept = model.cache_specs()
    assert all(type(s).__name__ == "CompositeSpec" and len(s.parts) == 2 for s in kept)
    first, second = kept[0].parts[0], kept[1].parts[0]
    assert (first.kv_heads, first.head_dim, first.window) == (1, 20, 7)  # both maps' key lanes side by side
    assert (second.kv_heads, second.head_dim, second.window) == (2, 10, 9)
    assert all(s.parts[1].shape == (40,) and s.parts[1].dtype == torch.float32 for s in kept)
    assert model.graph_safe


def test_parallel_block_with_parts_that_keep_their_products(engine):
    """A block whose mixer ends with a bias of its own cannot join the two output products: the parts run theirs, and the
    sum is the same."""
    engine("plain")
    from llmserve_triton_kernels_b200.parts.base import build_part, PartSpec

    torch.manual_seed(3)
    hid = 12
    common = {"hidden_size": hid, "num_heads": 2, "num_kv_heads": 1, "head_dim": 4, "value_dim": 4, "scale": 0.5, "rotary": {"dims": 4, "base": 10.0}, "window": 3}
    outs = []
    tensors = None
    for out_bias in (True, False):
        norm = lambda n: build_part("norm", PartSpec("rms_norm", {"size": hid, "eps": 1e-5, "weight_name": n}))  # noqa: E731
        parts = {"mixer_norm": norm("norm1"), "mixer": build_part("mixer", PartSpec("softmax_attention", {**common, "out_bias": out_bias})),
                 "ff_norm": norm("norm2"), "feed_forward": build_part("feed_forward", PartSpec("dense_mlp", {"hidden_size": hid, "intermediate_size": 8, "activation": "gelu"}))}
        block = build_part("block", PartSpec("parallel", {"hidden_size": hid, "token_shift": False}), **parts)
        if tensors is None:
            tensors = {role: {n: torch.randn([s for s in spec.shape]) * 0.3 for n, spec in p.tensors().items()} for role, p in parts.items()}
            tensors["mixer"]["o.b"].zero_()
        for role, p in parts.items():
            p.bind({n: tensors[role][n] for n in p.tensors()}, torch.float32, torch.device("cpu"))
        block.bind({}, torch.float32, torch.device("cpu"))
        assert (block.w_join is None) == out_bias
        from types import SimpleNamespace

        n = 5
        ctx = SimpleNamespace(num_tokens=n, num_requests=1, positions=torch.arange(n, dtype=torch.int32), cu_tokens=torch.tensor([0, n], dtype=torch.int32),
                              context_lens=torch.tensor([n], dtype=torch.int32), token_request=torch.zeros(n, dtype=torch.int32), shared={})
        cache = SimpleNamespace(pool=torch.zeros(2, 2, 1, 4, 4), page_table=torch.tensor([[1, 0]], dtype=torch.int32), slot_map=torch.tensor([4, 5, 6, 7, 0], dtype=torch.int32))
        x = torch.randn(n, hid, generator=torch.Generator().manual_seed(1))
        resid = x.clone()
        z = block.forward(resid, None, ctx, cache)
        outs.append(resid + z)
    assert torch.allclose(outs[0], outs[1], atol=1e-5)


# --------------------------------------------------------------------------------------------- generation and replay
@pytest.mark.parametrize("where", WHERE)
def test_greedy_generation_through_the_scheduler(where, engine, monkeypatch):
    """``LLM.generate`` with greedy sampling, several prompts at once in portions: every chosen token is the plain implementation's
    choice given the tokens before it (or its logit is within rounding of the best)."""
    engine(where)
    if where == "plain":
        from llmserve_triton_kernels_b200 import ops

        monkeypatch.setattr(ops, "argmax", plain_ops.argmax)
        monkeypatch.setattr(ops, "sample", plain_ops.sample)
    from llmserve_triton_kernels_b200.engine.llm import LLM
    from llmserve_triton_kernels_b200.sampling import SamplingParams
    from llmserve_triton_kernels_b200.weights.random_init import random_tensors

    cfg = configs.ODD
    device, dtype = ("cpu", "float32") if where == "plain" else ("cuda:0", where.split("-")[1])
    llm = LLM(cfg, dtype=dtype, device=device, seed=5, block_size=4, num_blocks=60, max_batch_size=3, chunk_size=6,
              max_num_batched_tokens=16, freeze_gc=False)
    tensors = random_tensors(llm.model.tensor_specs(), 5, 0.02, torch.bfloat16)
    prompts = list(tokens_for(cfg["vocab"], [5, 17, 9, 2], 8).values())
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12))
    assert [len(o.token_ids) for o in outs] == [12] * 4
    for prompt, o in zip(prompts, outs):
        logits = plain_pefedra.forward(cfg, tensors, prompt + o.token_ids)
        for k, tok in enumerate(o.token_ids):
            row = logits[len(prompt) + k - 1]
            slack = 1e-4 if dtype == "float32" else 0.05
            assert float(row.max() - row[tok]) <= slack * float(row.abs().max()), f"token {k} of a request is not the greedy choice"


@pytest.mark.parametrize("where", WHERE)
def test_preempted_requests_start_over(where, engine, monkeypatch):
    """A pool too small for all requests at once: some are preempted and recomputed, and every chosen token is still the greedy
    one (the shift's row and the pages start anew)."""
    engine(where)
    if where == "plain":
        from llmserve_triton_kernels_b200 import ops

        monkeypatch.setattr(ops, "argmax", plain_ops.argmax)
        monkeypatch.setattr(ops, "sample", plain_ops.sample)
    from llmserve_triton_kernels_b200.engine.llm import LLM
    from llmserve_triton_kernels_b200.sampling import SamplingParams
    from llmserve_triton_kernels_b200.weights.random_init import random_tensors

    cfg = configs.config([configs.layer(configs.turned(2, 1, 16, 16, 0.5, 400), 24), configs.layer(configs.differential(2, 1, 16, 16, 0.5, 400), 24)], width=32)
    device, dtype = ("cpu", "float32") if where == "plain" else ("cuda:0", where.split("-")[1])
    llm = LLM(cfg, dtype=dtype, device=device, seed=6, block_size=4, num_blocks=14, max_batch_size=3, chunk_size=8,
              max_num_batched_tokens=16, freeze_gc=False)
    tensors = random_tensors(llm.model.tensor_specs(), 6, 0.02, torch.bfloat16)
    prompts = list(tokens_for(cfg["vocab"], [9, 11, 7], 18).values())
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=16))
    assert llm.scheduler.stats.preemptions > 0
    for prompt, o in zip(prompts, outs):
        assert len(o.token_ids) == 16
        logits = plain_pefedra.forward(cfg, tensors, prompt + o.token_ids)
        for k, tok in enumerate(o.token_ids):
            row = logits[len(prompt) + k - 1]
            assert float(row.max() - row[tok]) <= (1e-4 if dtype == "float32" else 0.05) * float(row.abs().max())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program_as_a_user_starts_it(dtype, model_folder, tmp_path):
    """``bin/trace_run`` on a model folder: a mixed schedule over a pool that holds less than all requests together."""
    cfg = configs.ODD
    folder = model_folder(cfg, 31, torch.bfloat16, 0.1)
    from llmserve_triton_kernels_b200.weights.loader import read_safetensors

    tensors = read_safetensors(folder)
    reqs = tokens_for(cfg["vocab"], [70, 33, 5], 3)
    exp = expected_of(cfg, tensors, reqs)
    steps = [
        {"step": 0, "entries": [{"id": "r0", "tokens": reqs["r0"][:40], "want": [0, 39]}, {"id": "r2", "tokens": reqs["r2"], "want": [4]}], "end": ["r2"]},
        {"step": 1, "entries": [{"id": "r0", "tokens": reqs["r0"][40:69], "want": []}, {"id": "r1", "tokens": reqs["r1"][:2], "want": [1]}], "end": []},
        {"step": 2, "entries": [{"id": "r0", "tokens": reqs["r0"][69:], "want": [0]}, {"id": "r1", "tokens": reqs["r1"][2:], "want": [0, 30]}], "end": ["r0", "r1"]},
    ]
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900, env={**os.environ})
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [line for line in proc.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    vocab = cfg["vocab"]
    rows = {n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, vocab) for n in (0, 1, 2)}
    got = {("r0", 0): rows[0][0], ("r0", 39): rows[0][1], ("r2", 4): rows[0][2], ("r1", 1): rows[1][0], ("r0", 69): rows[2][0], ("r1", 2): rows[2][1],
           ("r1", 32): rows[2][2]}
    check(got, exp, dtype, "replay")

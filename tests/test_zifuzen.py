"""The Zifuzen design in the engine against the plain implementation (tests/plain_zifuzen.py).

Every test makes its own small configuration and random weights.  The engine runs the requests in some way of cutting the work
(whole, token by token, in portions down to two tokens, in mixed batches over a pool so small that pages and state slots are used
again) and the logits at every position are compared with the plain implementation's, which knows no cache.  On the GPU the
engine's kernels run, in true 32-bit and in bfloat16; without one the same host logic runs over the plain operations.
"""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_ops
import plain_zifuzen
import zifuzen_configs as configs
from test_kafepel import Driver, engine, make_model, tokens_for  # noqa: F401  (the same harness; ``engine`` is a fixture)
from test_kafepel import BF16_TOL, F32_TOL
from test_nudodra import _scale_of

WHERE = ["plain", pytest.param("cuda-float32", marks=pytest.mark.gpu), pytest.param("cuda-bfloat16", marks=pytest.mark.gpu)]
ROOT = Path(__file__).resolve().parent.parent


def expected_of(cfg, tensors, requests):
    return {r: plain_zifuzen.forward(cfg, tensors, t) for r, t in requests.items()}


def check(got, expected, dtype, what="", cfg=None):
    """A row's error is measured against the row's size (in bfloat16: at least the size of all rows).  In 32-bit one row in ten (or
    one) may be beyond the tolerance, by no more than ``most``: where a query or key is almost nothing before it becomes a unit vector,
    or a part's result almost nothing before its norm, rounding is magnified and nothing is wrong.  In bfloat16 it may also move a
    router's choice between two experts of almost equal score, after which a request's later rows differ a little as well: one row in
    four, and more room for the odd configuration's heads of a few lanes."""
    tol, most = (F32_TOL, 20 * F32_TOL) if dtype == "float32" else (0.15 if cfg is configs.ODD else BF16_TOL, 2.0)
    allowed = max(1, len(got) // (10 if dtype == "float32" else 4))
    floor = _scale_of([expected[r.split("#")[0]][pos] for r, pos in got], dtype)
    over = []
    for (req, pos), row in sorted(got.items()):
        ref = expected[req.split("#")[0]][pos].float()
        assert torch.isfinite(row).all(), f"{what}: non-finite logits at request {req!r} position {pos}"
        d = row - ref
        err = float((d - d.mean()).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(floor))
        assert err <= most, f"{what}: request {req!r} position {pos} is wrong: error {err:.3e}"
        if err > tol:
            over.append((req, pos, err))
    assert len(over) <= allowed, f"{what}: {len(over)} of {len(got)} rows are beyond {tol:.1e}; the first: {over[0]}"


def _loud(tensors):
    """Weights that random draws would leave near nothing, or near one another, made so that leaving them out shows: positions,
    biases, decays from slow to fast, step sizes on both sides of a half, corrections that move choices, norms away from one,
    output matrices large enough for the cap to bend the logits, expert products that pass their bounds."""
    g = torch.Generator().manual_seed(99)
    for name, t in tensors.items():
        normal = lambda std, mean=0.0: (mean + torch.randn(t.shape, generator=g) * std).to(t.dtype)  # noqa: E731,B023
        end = name.rsplit(".", 1)[-1]
        if name == "embed":
            tensors[name] = normal(0.4)
        elif name == "pos":
            tensors[name] = normal(0.8)
        elif name == "head":
            tensors[name] = normal(8.0 * t.shape[1] ** -0.5)
        elif end == "A_log":
            tensors[name] = (torch.rand(t.shape, generator=g) * 4.0 - 3.0).to(t.dtype)
        elif end == "dt_bias":
            tensors[name] = normal(1.0, -1.0)
        elif name.endswith((".mix.a", ".mix.b")):
            tensors[name] = normal(1.5 * t.shape[1] ** -0.5)
        elif end == "b" and name.count(".") == 3:  # biases of the dense feed-forward
            tensors[name] = normal(0.4)
        elif end == "correction":
            tensors[name] = normal(1.5)
        elif end == "conv":
            tensors[name] = normal(0.6)
        elif name.endswith(("q.norm", "k.norm")):
            tensors[name] = normal(0.3, 1.5)
        elif end in ("norm", "norm1", "norm2"):
            tensors[name] = normal(0.3, 1.0)
        elif end in ("q", "k", "v", "g", "gate", "up", "router"):
            tensors[name] = normal(1.5 * t.shape[1] ** -0.5)


# --------------------------------------------------------------------------------------------- the plain statement
def test_plain_mechanisms_one_by_one():
    """The oracle's own parts against what they are by definition, on inputs where the answer is known."""
    f64, P = torch.float64, plain_zifuzen
    tensor = lambda x: torch.tensor(x, dtype=f64)  # noqa: E731
    y = P.layer_norm(tensor([[1.0, 3.0]]), 0.0, tensor([1.0, 5.0]))
    assert y.tolist() == [[-1.0, 5.0]]
    assert torch.allclose(P.layer_norm(tensor([[1.0, 3.0]]), 3.0, tensor([1.0, 1.0])), tensor([[-0.5, 0.5]]))
    W = {"embed": tensor([[1.0], [2.0]]), "pos": tensor([[10.0], [20.0], [30.0]])}
    assert P.embedding(W, [1, 0], 3.0).tolist() == [[16.0], [23.0]]
    u, w = tensor([[1.0], [10.0], [100.0]]), tensor([[5.0, 2.0]])
    assert P.short_conv(u, w).tolist() == [[2.0], [25.0], [250.0]]
    assert torch.allclose(P.unit(tensor([[3.0, 4.0]])), tensor([[0.6, 0.8]]), atol=1e-6)
    # the rule on one head and lane: forget, read at the key, correct, read out with the new write
    q, k, v = tensor([[[2.0]], [[3.0]]]), tensor([[[1.0]], [[0.5]]]), tensor([[[4.0]], [[8.0]]])
    o = P.delta_recurrence(q, k, v, tensor([[0.5], [0.25]]), tensor([[0.0], [math.log(0.5)]]))
    s1 = 0.5 * 4.0
    s2 = 0.5 * s1 + 0.5 * (0.25 * (8.0 - 0.5 * s1 * 0.5))
    assert torch.allclose(o.flatten(), tensor([2.0 * s1, 3.0 * s2]))
    W = {"a": tensor([[1.0]]), "dt_bias": tensor([0.5]), "A_log": tensor([math.log(2.0)]), "b": tensor([[1.0]])}
    assert torch.allclose(P.log_decays(tensor([[0.0]]), W, ""), tensor([[-2.0 * math.log(1.0 + math.exp(0.5))]]))
    assert torch.allclose(P.step_sizes(tensor([[0.0]]), W, ""), tensor([[0.5]]))
    # groups: (0.9 + 0.1) against (0.6 + 0.55): the group of the single best expert loses; negative choice scores can win
    W = {"router": torch.eye(4, dtype=f64) * 1.0, "correction": tensor([0.0, 0.0, 0.0, 0.0])}
    z = torch.logit(tensor([[0.9, 0.1, 0.6, 0.55]]))
    w = P.router_weights(z, W, "", {"experts": 4, "top": 1, "scale": 2.0, "groups": {"count": 2, "keep": 1}})
    assert torch.allclose(w, tensor([[0.0, 0.0, 2.0, 0.0]]))
    W["correction"] = tensor([-3.0, -3.0, -5.0, -5.0])
    w = P.router_weights(z, W, "", {"experts": 4, "top": 2, "scale": 1.0, "groups": {"count": 2, "keep": 1}})
    assert torch.allclose(w, tensor([[0.9, 0.1, 0.0, 0.0]]))
    W = {"gate": tensor([[1.0]]), "up": tensor([[1.0]]), "down": tensor([[1.0]])}
    s = lambda x: 1.0 / (1.0 + math.exp(-x))  # noqa: E731
    y = P.bounded_expert(tensor([[9.0], [-9.0]]), W, "", 2.0)
    assert torch.allclose(y, tensor([[2.0 * s(3.404) * 3.0], [-9.0 * s(-9.0 * 1.702) * -1.0]]))
    assert torch.allclose(P.soft_cap(tensor([0.0, 1e9, -2.0]), 5.0), tensor([0.0, 5.0, 5.0 * math.tanh(-0.4)]))
    assert torch.allclose(P.gelu_tanh(tensor([0.0, 1.0, -1.0])), tensor([0.0, 0.8411919906, -0.1588080094]))


# --------------------------------------------------------------------------------------------- mechanisms alone
ALONE = {
    "delta": configs.config([configs.layer(configs.delta(6, 2, 10, 7, 3))], width=32),
    "delta_16": configs.config([configs.layer(configs.delta(4, 4, 16, 16, 4, "delta_2"))], width=32),
    "delta_64": configs.config([configs.layer(configs.delta(2, 1, 64, 48, 2))], width=48),
    "delta_long_keys": configs.config([configs.layer(configs.delta(2, 2, 160, 33, 4))], width=48),
    "delta_many_lanes": configs.config([configs.layer(configs.delta(2, 1, 256, 96, 4))], width=48),
    "one_tap": configs.config([configs.layer(configs.delta(3, 1, 12, 20, 1))], width=32),
    "sixteen_taps": configs.config([configs.layer(configs.delta(3, 3, 12, 20, 16))], width=32),
    "attention": configs.config([configs.layer(configs.attention(6, 2, 10, 6, 0.7))], width=32),
    "attention_48": configs.config([configs.layer(configs.attention(8, 2, 48, 32, 0.4))], width=64),
    "shared_pages": configs.config([configs.layer(configs.attention(2, 1, 16, 32, 0.5)), configs.layer(configs.attention(4, 1, 16, 32, 0.3, kv_from=0))], width=48),
    "dense": configs.config([configs.layer(configs.attention(1, 1, 4, 4, 0.5), configs.dense(40))], width=32),
    "mixture": configs.config([configs.layer(configs.attention(1, 1, 16, 16, 0.5), configs.moe(12, 3, 16, 0.8, groups=(4, 2), shared=(32, 0.5)))], width=64),
    "mixture_odd": configs.config([configs.layer(configs.attention(1, 1, 4, 4, 0.5), configs.moe(9, 2, 5, 1.2, groups=(3, 1)))], width=30),
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
    check(d.got, exp, dtype, "whole", cfg)
    d.got.clear()
    for i, t in enumerate(reqs["r0"]):
        d.run([("r0", [t])], end=["r0"] if i == len(reqs["r0"]) - 1 else [])
    check(d.got, exp, dtype, "token by token", cfg)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_residual_stream_after_every_layer(name, where, engine):
    engine(where)
    cfg = configs.ALL[name]
    model, tensors, dtype = make_model(cfg, 3, where, change=_loud)
    tokens = tokens_for(cfg["vocab"], [19], 2)["r0"]
    _, layers = plain_zifuzen.forward(cfg, tensors, tokens, return_layers=True)
    seen = []
    model.layer_probe = lambda i, x: seen.append(x.float().cpu().clone())
    Driver(model, num_pages=16).run([("r0", tokens)], end=["r0"])
    assert len(seen) == len(layers) == len(cfg["layers"])
    tol = 3e-4 if dtype == "float32" else 8e-2
    for i, x in enumerate(seen):
        scale = float(layers[i].abs().max())
        over = (x - layers[i].float()).abs().amax(-1) > tol * scale
        # in bfloat16 rounding may move a router's choice between two experts of almost equal score
        assert int(over.sum()) <= (0 if dtype == "float32" else 2), f"the stream differs after layer {i}"


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
    check(d.got, exp, dtype, "whole", cfg)
    d.got.clear()
    t = reqs["r3"]
    d.run([("r3", t[:40])])
    for i in range(40, len(t)):
        d.run([("r3", [t[i]])], end=["r3"] if i == len(t) - 1 else [])
    check(d.got, exp, dtype, "decode", cfg)
    d.got.clear()
    for r in ("r2", "r3"):
        t, i, k = reqs[r], 0, 0
        sizes = (1, 2, 7, 2, 18, 3, 5, 2, 1, 9)
        while i < len(t):
            n = min(sizes[k % len(sizes)], len(t) - i)
            d.run([(r, t[i : i + n])], end=[r] if i + n == len(t) else [])
            i, k = i + n, k + 1
    check(d.got, exp, dtype, "portions", cfg)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_mixed_batches_with_pages_and_slots_used_again(name, where, engine):
    """Up to four unequal requests a step, portions beside single tokens, over a pool of few pages and four state slots: every
    request's logits equal those of the request alone, also on pages and slots that others gave back (a slot's matrices and the
    convolutions' rows must start at zero again)."""
    engine(where)
    cfg = configs.ALL[name]
    model, tensors, dtype = make_model(cfg, 17, where, change=_loud)
    base = tokens_for(cfg["vocab"], [50, 9, 31, 64, 3, 40], 21)
    exp = expected_of(cfg, tensors, base)
    reqs = {**base, **{r + "#2": t for r, t in base.items()}}  # each once more, on used pages and slots
    prefill = {r: max(1, len(t) - 6) for r, t in reqs.items()}
    d = Driver(model, num_pages=52, page_size=4, max_requests=4)
    waiting, live, turn = list(reqs), {}, 0
    while waiting or live:
        if waiting and len(live) < 4:
            live[waiting.pop(0)] = 0
        entries, end = [], []
        turn += 1
        for r, fed in list(live.items()):
            t = reqs[r]
            n = min(19 if turn % 3 == 0 else 7, prefill[r] - fed) if fed < prefill[r] else 1
            n = min(n, len(t) - fed)
            entries.append((r, t[fed : fed + n]))
            live[r] = fed + n
            if live[r] == len(t):
                end.append(r)
                del live[r]
        d.run(entries, end=end)
    assert len({k[0] for k in d.got}) == len(reqs)
    check(d.got, exp, dtype, "mixed", cfg)
    assert d.cache.slots.num_used == 0 and all(g.allocator.num_used == 0 for g in d.cache.groups)


@pytest.mark.parametrize("where", WHERE)
def test_a_request_left_out_of_steps_goes_on_where_it_was(where, engine):
    """A request that sits out steps while another takes a slot, steps and ends: its matrices, rows and pages are as it left them."""
    engine(where)
    cfg = configs.ODD
    model, tensors, dtype = make_model(cfg, 7, where, change=_loud)
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
    check(d.got, exp, dtype, "left out and taken up again", cfg)


@pytest.mark.parametrize("where", WHERE)
def test_long_decoding(where, engine):
    """A short prompt, then many tokens one by one: pages fill one after the other, the matrices and rows move on at every step."""
    engine(where)
    cfg = configs.ODD
    model, tensors, dtype = make_model(cfg, 17, where, change=_loud)
    t = tokens_for(cfg["vocab"], [150], 4)["r0"]
    exp = expected_of(cfg, tensors, {"r0": t})
    d = Driver(model, num_pages=84, page_size=4)
    d.run([("r0", t[:3])])
    for i in range(3, len(t)):
        d.run([("r0", [t[i]])], end=["r0"] if i == len(t) - 1 else [])
    check(d.got, exp, dtype, "long decoding", cfg)


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
    check(d.got, exp, dtype, "whole", cfg)
    d.got.clear()
    d.run([("r1", reqs["r1"][:39])])
    d.run([("r0", reqs["r0"][:150]), ("r1", reqs["r1"][39:])], end=["r1"])
    d.run([("r0", reqs["r0"][150:320])])
    for i in range(320, 330):
        d.run([("r0", [reqs["r0"][i]])], end=["r0"] if i == 329 else [])
    check(d.got, exp, dtype, "two long portions, then single tokens", cfg)


# --------------------------------------------------------------------------------------------- faults that random weights would hide
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("dim", [16, 10])
def test_one_far_key_decides(where, dim, engine):
    """Attention with scores so sharp that a query leans on the one key it looks for: an embedding is two codes side by side, W_k
    reads the first and W_q the second, and token i's second code is token 40 + i's first.  The token looked for stands once, more
    than a hundred places back and on every side of page borders in turn; the plain statement without it differs visibly.  A prompt
    in portions that end inside pages, then single tokens."""
    engine(where)
    half = 16
    cfg = configs.config([configs.layer(configs.attention(2, 1, dim, dim, 3.0)), configs.layer(configs.attention(2, 1, dim, dim, 3.0, kv_from=0))],
                         width=2 * half, vocab=128, scale=1.0)

    def codes(tensors):
        _loud(tensors)
        g = torch.Generator().manual_seed(5)
        first, second = torch.randn(128, half, generator=g), torch.randn(128, half, generator=g)
        second[:40] = first[40:80]
        reads, none = torch.randn(dim, half, generator=g), torch.zeros(dim, half)
        put = {"embed": torch.cat((first, second), 1), "pos": torch.zeros(cfg["max_positions"], 2 * half), "l0.mix.k": torch.cat((reads, none), 1),
               "l0.mix.q": torch.cat((none, reads), 1).repeat(2, 1), "l0.mix.q.norm": torch.ones(dim), "l0.mix.k.norm": torch.ones(dim)}
        tensors.update({n: t.to(torch.bfloat16) for n, t in put.items()})

    model, tensors, dtype = make_model(cfg, 29, where, std=0.3, change=codes)
    t = torch.randint(80, 128, (260,), generator=torch.Generator().manual_seed(3)).tolist()
    for i in range(40):
        t[3 * i + i % 3] = 40 + i
        t[140 + 3 * i] = i
    exp = expected_of(cfg, tensors, {"r0": t})
    for i in (0, 7, 20, 39):
        without = list(t)
        without[3 * i + i % 3] = 127
        far = plain_zifuzen.forward(cfg, tensors, without)[140 + 3 * i] - exp["r0"][140 + 3 * i]
        assert float(far.pow(2).mean().sqrt()) > 0.2 * float(exp["r0"].pow(2).mean().sqrt())
    d = Driver(model, num_pages=70, page_size=4)
    i = 0
    for n in (3, 126, 2, 70, 39):
        d.run([("r0", t[i : i + n])])
        i += n
    for j in range(i, len(t)):
        d.run([("r0", [t[j]])], end=["r0"] if j == len(t) - 1 else [])
    check(d.got, exp, dtype, "a far key", cfg)


@pytest.mark.parametrize("where", WHERE)
def test_a_slow_state_remembers_far_tokens(where, engine):
    """Decays so slow that the state after hundreds of tokens still holds the first: a different first token moves the last logits,
    however the tokens were cut (portions that end inside the scan's blocks of eight, then single tokens)."""
    engine(where)
    cfg = configs.config([configs.layer(configs.delta(2, 1, 48, 20, 3)), configs.layer(configs.delta(2, 2, 16, 16, 2, "delta_2"))], width=32)

    def slow(tensors):
        _loud(tensors)
        for name, t in tensors.items():
            if name.endswith("A_log"):
                tensors[name] = torch.full_like(t, -7.0)
            elif name.endswith(".mix.b"):
                tensors[name] = (t.float() - 0.5).to(t.dtype)

    model, tensors, dtype = make_model(cfg, 37, where, std=0.3, change=slow)
    t = tokens_for(cfg["vocab"], [220], 14)["r0"]
    exp = expected_of(cfg, tensors, {"r0": t})
    other = [(t[0] + 1) % cfg["vocab"]] + t[1:]
    moved = plain_zifuzen.forward(cfg, tensors, other)[-20:] - exp["r0"][-20:]
    assert float(moved.abs().max()) > 0.02
    d = Driver(model, num_pages=70, page_size=4)
    i = 0
    for n in (2, 17, 33, 5, 90, 24, 19):
        d.run([("r0", t[i : i + n])])
        i += n
    for j in range(i, len(t)):
        d.run([("r0", [t[j]])], end=["r0"] if j == len(t) - 1 else [])
    check(d.got, exp, dtype, "a slow state", cfg)


@pytest.mark.parametrize("what", ["positions", "embedding scale", "mean", "conv", "unit", "decay", "step size", "gate", "head norm", "own write", "qk norm",
                                  "shared pages", "bias", "correction", "groups", "shared expert", "limit", "shift", "router scale", "cap"])
def test_every_mechanism_shows_in_the_plain_statement(what, monkeypatch):
    """The weights of these tests are such that leaving a mechanism out moves the plain statement's logits by far more than any
    tolerance here: what the engine is compared with would not forgive it."""
    cfg = json.loads(json.dumps(configs.ODD))
    model, tensors, _ = make_model(cfg, 7, "plain", change=_loud)
    t = tokens_for(cfg["vocab"], [45], 9)["r0"]
    right = plain_zifuzen.forward(cfg, tensors, t)
    tensors = dict(tensors)
    P = plain_zifuzen
    zero = lambda *ends: {n: (torch.zeros_like(x) if n.endswith(ends) else x) for n, x in tensors.items()}  # noqa: E731
    one = lambda *ends: {n: (torch.ones_like(x) if n.endswith(ends) else x) for n, x in tensors.items()}  # noqa: E731
    mlps = [layer["mlp"] for layer in cfg["layers"] if layer["mlp"] and layer["mlp"]["kind"] == "moe"]
    if what == "positions":
        tensors["pos"] = torch.zeros_like(tensors["pos"])
    elif what == "embedding scale":
        cfg["embedding"]["scale"] = 1.0
    elif what == "mean":
        monkeypatch.setattr(P, "layer_norm", lambda x, eps, w: P.rms(x, eps, w))
    elif what == "conv":
        monkeypatch.setattr(P, "short_conv", lambda u, w: u * w[:, -1])
    elif what == "unit":
        monkeypatch.setattr(P, "unit", lambda x: x)
    elif what == "decay":
        monkeypatch.setattr(P, "log_decays", lambda h, W, p: torch.zeros(h.shape[0], W[p + "a"].shape[0], dtype=h.dtype))
    elif what == "step size":
        monkeypatch.setattr(P, "step_sizes", lambda h, W, p: torch.ones(h.shape[0], W[p + "b"].shape[0], dtype=h.dtype))
    elif what == "gate":
        tensors = one("mix.g")
    elif what == "head norm":
        tensors = one("mix.norm")
    elif what == "own write":  # the read-out in front of the token's own write
        rule = P.delta_recurrence
        shifted = lambda x: torch.cat((torch.zeros_like(x[:1]), x[:-1]))  # noqa: E731
        monkeypatch.setattr(P, "delta_recurrence", lambda q, k, v, b, g: rule(q, shifted(k), shifted(v), shifted(b), shifted(g)))
    elif what == "qk norm":
        tensors = one("q.norm", "k.norm")
    elif what == "shared pages":
        cfg["layers"][4]["mixer"].update(kv_from=3, kv_heads=3, heads=3)
        tensors = {n: (torch.randn(36, 40) if n == "l4.mix.q" else torch.randn(12) if n == "l4.mix.q.norm" else torch.randn(40, 42) if n == "l4.mix.o" else x)
                   for n, x in tensors.items()}
        cfg["layers"][4]["mixer"].update(dim=12, vdim=14)
    elif what == "bias":
        tensors = zero("mlp.gate.b")
    elif what == "correction":
        tensors = zero("correction")
    elif what == "groups":
        for m in mlps:
            m["router"].pop("groups", None)
    elif what == "shared expert":
        for m in mlps:
            m.pop("shared", None)
    elif what == "limit":
        for m in mlps:
            m["expert"]["limit"] = 1e9
    elif what == "shift":
        monkeypatch.setattr(P, "bounded_expert", lambda h, W, p, limit: (P.silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T)
    elif what == "router scale":
        for m in mlps:
            m["router"]["scale"] *= 2.0
    else:
        monkeypatch.setattr(P, "soft_cap", lambda z, cap: z)
    wrong = P.forward(cfg, tensors, t)
    d = wrong - right
    assert float((d - d.mean(-1, keepdim=True)).pow(2).mean().sqrt() / right.pow(2).mean().sqrt()) > 0.05


# --------------------------------------------------------------------------------------------- configuration and plan
def test_configuration_round_trip_and_errors():
    from llmserve_triton_kernels_b200.config import ConfigError, ZifuzenConfig, architecture_of

    for cfg in configs.ALL.values():
        typed = architecture_of(cfg).config_class.from_dict(cfg)
        assert isinstance(typed, ZifuzenConfig) and typed.to_dict() == cfg
        assert ZifuzenConfig.from_dict(typed.to_dict()) == typed
    for path, value, match in (
        (("layers", 0, "mixer", "conv"), 0, "conv"), (("layers", 0, "mixer", "conv"), 17, "taps"), (("layers", 0, "mixer", "kv_heads"), 4, "multiple"),
        (("layers", 2, "type"), "retention", "retention"), (("layers", 0, "mlp", "kind"), "sparse", "sparse"), (("layers", 4, "mixer", "kv_from"), 2, "own"),
        (("layers", 4, "mixer", "kv_from"), 5, "earlier"), (("layers", 4, "mixer", "vdim"), 5, "vdim"), (("layers", 1, "mixer", "scale"), None, "scale"),
        (("layers", 1, "mlp", "router", "groups", "count"), 4, "groups"), (("layers", 1, "mlp", "router", "groups", "keep"), 4, "groups"),
        (("layers", 3, "mlp", "router", "top"), 6, "groups"), (("layers", 1, "mlp", "shared", "limit"), None, "limit"), (("width",), None, "width"),
        (("max_positions",), None, "max_positions"), (("logit_softcap",), -1.0, "softcap"),
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
            ZifuzenConfig.from_dict(bad)


def test_plan_names_every_tensor_of_the_design_and_what_layers_keep():
    model, _, _ = make_model(configs.ODD, 1, "plain")
    specs = model.tensor_specs()
    shapes = {
        "embed": (97, 40), "pos": (400, 40), "head": (97, 40), "final.norm": (40,), "l0.norm1": (40,), "l0.norm2": (40,), "l0.mix.q": (20, 40),
        "l0.mix.q.conv": (20, 3), "l0.mix.k.conv": (20, 3), "l0.mix.v": (42, 40), "l0.mix.v.conv": (42, 3), "l0.mix.b": (6, 40), "l0.mix.a": (6, 40),
        "l0.mix.A_log": (6,), "l0.mix.dt_bias": (6,), "l0.mix.norm": (7,), "l0.mix.g": (42, 40), "l0.mix.o": (40, 42), "l0.mlp.gate.b": (28,),
        "l0.mlp.down": (40, 28), "l0.mlp.down.b": (40,), "l1.mix.q": (60, 40), "l1.mix.k": (20, 40), "l1.mix.v": (12, 40), "l1.mix.q.norm": (10,),
        "l1.mix.k.norm": (10,), "l1.mlp.router": (6, 40), "l1.mlp.correction": (6,), "l1.mlp.e5.down": (40, 9), "l1.mlp.shared.up": (11, 40),
        "l4.mix.q": (40, 40), "l4.mix.q.norm": (10,), "l4.mix.o": (40, 24),
    }
    for name, shape in shapes.items():
        assert specs[name].shape == shape, name
    for name in ("l2.norm2", "l2.mlp.up", "l3.mlp.shared.up", "l4.mix.k", "l4.mix.k.norm", "l4.mix.v", "l1.mlp.router.b"):
        assert name not in specs, name
    kept = model.cache_specs()
    assert [s.shape for s in kept[0].parts] == [(6, 10, 7), (2, 82)] and all(s.dtype == torch.float32 for s in kept[0].parts)
    assert (kept[1].kv_heads, kept[1].head_dim, kept[1].window) == (2, 10, None) and kept[4] is None
    assert model.graph_safe


def test_positions_beyond_the_table_are_refused(engine):
    engine("plain")
    cfg = configs.config([configs.layer(configs.attention(1, 1, 4, 4, 0.5))], width=8, places=20)
    model, _, _ = make_model(cfg, 1, "plain")
    d = Driver(model, num_pages=24)
    d.run([("r0", [1] * 20)])
    with pytest.raises(ValueError, match="20 positions"):
        d.run([("r0", [1])])


# --------------------------------------------------------------------------------------------- generation and replay
def _greedy(where, monkeypatch, cfg, seed, lengths, new, **engine_args):
    """Generates greedily; every chosen token is the plain statement's choice given the tokens before it (or its logit is within
    rounding of the best)."""
    if where == "plain":
        from llmserve_triton_kernels_b200 import ops

        monkeypatch.setattr(ops, "argmax", plain_ops.argmax)
        monkeypatch.setattr(ops, "sample", plain_ops.sample)
    from llmserve_triton_kernels_b200.engine.llm import LLM
    from llmserve_triton_kernels_b200.sampling import SamplingParams
    from llmserve_triton_kernels_b200.weights.random_init import random_tensors

    device, dtype = ("cpu", "float32") if where == "plain" else ("cuda:0", where.split("-")[1])
    llm = LLM(cfg, dtype=dtype, device=device, seed=seed, block_size=4, max_batch_size=3, max_num_batched_tokens=16, freeze_gc=False, **engine_args)
    tensors = random_tensors(llm.model.tensor_specs(), seed, 0.02, torch.bfloat16)
    prompts = list(tokens_for(cfg["vocab"], lengths, 8).values())
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=new))
    assert [len(o.token_ids) for o in outs] == [new] * len(prompts)
    for prompt, o in zip(prompts, outs):
        logits = plain_zifuzen.forward(cfg, tensors, prompt + o.token_ids)
        for k, tok in enumerate(o.token_ids):
            row = logits[len(prompt) + k - 1]
            slack = 1e-4 if dtype == "float32" else 0.05
            assert float(row.max() - row[tok]) <= slack * float(row.abs().max()), f"token {k} of a request is not the greedy choice"
    return llm


@pytest.mark.parametrize("where", WHERE)
def test_greedy_generation_through_the_scheduler(where, engine, monkeypatch):
    """``LLM.generate`` with greedy sampling, several prompts at once in portions."""
    engine(where)
    _greedy(where, monkeypatch, configs.ODD, 5, [5, 17, 9, 2], 12, num_blocks=60, chunk_size=6)


@pytest.mark.parametrize("where", WHERE)
def test_preempted_requests_start_over(where, engine, monkeypatch):
    """A pool too small for all requests at once: some are preempted and recomputed, and every chosen token is still the greedy
    one (the matrices, the convolutions' rows and the pages start anew)."""
    engine(where)
    cfg = configs.config([configs.layer(configs.attention(2, 1, 16, 16, 0.5), configs.dense(24)), configs.layer(configs.delta(2, 1, 16, 16, 3), configs.dense(24))], width=32)
    llm = _greedy(where, monkeypatch, cfg, 6, [9, 11, 7], 16, num_blocks=14, chunk_size=8)
    assert llm.scheduler.stats.preemptions > 0


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
    check(got, exp, dtype, "replay", cfg)

"""The kernels that the Zifuzen design added or widened against their plain statements (tests/plain_ops.py) at odd sizes: the gated
delta rule in its two forms (few tokens: a head's state in registers; prompts: blocks of eight tokens), the norm behind a part, the
embedding with positions, the convolution with silu behind it, the gated activation with gelu, the cap on logits, the router with
sigmoid scores and groups of experts."""

from __future__ import annotations

from types import SimpleNamespace

import pytest
import torch

import plain_ops
from test_kafepel_kernels_gpu import DEV, _ops, close

pytestmark = pytest.mark.gpu


def batch(counts):
    cu = [0]
    for c in counts:
        cu.append(cu[-1] + c)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)  # noqa: E731
    return SimpleNamespace(num_tokens=cu[-1], num_requests=len(counts), max_query_len=max(counts), cu_tokens=i32(cu),
                           token_request=i32([r for r, c in enumerate(counts) for _ in range(c)]), host_cu_tokens=cu)


# heads, kv heads, key lanes, value lanes
SIZES = [(6, 2, 10, 7), (1, 1, 1, 1), (4, 4, 32, 32), (3, 1, 64, 128), (8, 4, 48, 80), (2, 1, 128, 64), (2, 2, 130, 36), (5, 5, 200, 24), (2, 1, 256, 96), (4, 1, 3, 65)]


def delta_inputs(H, G, D, V, n, slots, seed, slow=False):
    g = torch.Generator(device=DEV).manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)  # noqa: E731
    pad = 3  # columns behind the last: rows have a pitch
    y = rnd(n, 2 * G * D + H * V + pad)
    proj = rnd(n, H * V + 2 * H + pad)
    a_log = torch.full((H,), -8.0, device=DEV) if slow else rnd(H) - 0.5
    states = rnd(slots, H, D, V) * 0.3
    return dict(y=y, beta=proj[:, H * V : H * V + H], decay=proj[:, H * V + H : H * V + 2 * H], a_log=a_log, dt_bias=rnd(H), gate=proj[:, : H * V],
                weight=1.0 + 0.3 * rnd(V), states=states)


def run_delta(ops, x, slots, ctx, H, G, D, V, dtype=torch.float32):
    y, states = x["y"].clone(), x["states"].clone()
    out = ops.delta_rule(y, x["beta"], x["decay"], x["a_log"], x["dt_bias"], x["gate"], x["weight"], 1e-5, states, slots, ctx, heads=H, kv_heads=G, dim=D,
                         value_dim=V, out_dtype=dtype)
    return out, states


@pytest.mark.parametrize("counts", [[1], [1, 1, 1], [3, 16, 1], [8], [9, 1, 40, 7], [64, 1], [130, 2, 17]])
@pytest.mark.parametrize("H,G,D,V", SIZES)
def test_delta_rule_against_plain(H, G, D, V, counts):
    ops, ctx = _ops(), batch(counts)
    x = delta_inputs(H, G, D, V, ctx.num_tokens, len(counts) + 2, D + V)
    slots = torch.arange(len(counts), 0, -1, dtype=torch.int32, device=DEV)
    want, want_states = run_delta(plain_ops, x, slots, ctx, H, G, D, V)
    got, states = run_delta(ops, x, slots, ctx, H, G, D, V)
    close(got, want, 5e-4, "rows")  # a head whose o is almost nothing is normed up
    close(states, want_states, 2e-5, "states")
    rough, _ = run_delta(ops, x, slots, ctx, H, G, D, V, torch.bfloat16)
    close(rough.float(), want, 1e-2, "rows in bfloat16")


@pytest.mark.parametrize("wide", [False, True])
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 32, 96), (2, 1, 64, 130), (3, 3, 100, 64), (2, 2, 128, 40)])
def test_delta_scan_with_few_and_many_columns_a_cta(H, G, D, V, wide, monkeypatch):
    ops = _ops()
    monkeypatch.setattr(ops, "_sm_count", lambda: 1 if wide else 10000)
    ctx = batch([37, 200, 1])
    x = delta_inputs(H, G, D, V, ctx.num_tokens, 3, 5)
    slots = torch.tensor([2, 0, 1], dtype=torch.int32, device=DEV)
    want, want_states = run_delta(plain_ops, x, slots, ctx, H, G, D, V)
    got, states = run_delta(ops, x, slots, ctx, H, G, D, V)
    close(got, want, 5e-4, "rows")
    close(states, want_states, 2e-5, "states")


@pytest.mark.parametrize("H,G,D,V", [(2, 1, 64, 48), (1, 1, 16, 16)])
def test_delta_rule_forms_agree_over_a_long_slow_sequence(H, G, D, V):
    """Decays near one: what the first tokens wrote is still there at the end.  The prompt in one scan, in portions that end inside
    blocks, and token by token through the form for few tokens."""
    ops, n = _ops(), 300
    x = delta_inputs(H, G, D, V, n, 1, 9, slow=True)
    x["states"].zero_()
    slots = torch.zeros(1, dtype=torch.int32, device=DEV)
    want, want_states = run_delta(plain_ops, x, slots, batch([n]), H, G, D, V)

    def cut(sizes):
        states, rows, i = x["states"].clone(), [], 0
        for size in sizes:
            part = {k: (v[i : i + size] if k in ("y", "beta", "decay", "gate") else v) for k, v in x.items()}
            out, states = run_delta(ops, {**part, "states": states}, slots, batch([size]), H, G, D, V)
            rows.append(out)
            i += size
        return torch.cat(rows), states

    for sizes in ([n], [17, 3, 100, 21, 2, 57, 100], [1] * n):
        got, states = cut(sizes)
        close(got, want, 1e-3, f"rows of {len(sizes)} portions")
        close(states, want_states, 1e-4, f"states of {len(sizes)} portions")


def test_delta_rule_with_equal_keys_and_strong_corrections():
    """Every token has the same key and step sizes near one: the state is overwritten again and again, the triangular systems of the
    blocks are at their worst conditioned; and decays so fast that nothing is left after a token."""
    ops, H, G, D, V = _ops(), 2, 1, 32, 32
    ctx = batch([90])
    slots = torch.zeros(1, dtype=torch.int32, device=DEV)
    for fast in (False, True):
        x = delta_inputs(H, G, D, V, 90, 1, 3)
        x["y"][:, G * D : 2 * G * D] = x["y"][:1, G * D : 2 * G * D]
        x["beta"].fill_(9.0)
        x["a_log"].fill_(6.0 if fast else -9.0)
        want, want_states = run_delta(plain_ops, x, slots, ctx, H, G, D, V)
        got, states = run_delta(ops, x, slots, ctx, H, G, D, V)
        close(got, want, 1e-3, "rows")
        close(states, want_states, 1e-4, "states")


@pytest.mark.parametrize("center", [True, False])
@pytest.mark.parametrize("n,c", [(1, 64), (5, 40), (3, 7), (2, 2048), (700, 192), (400, 2048), (300, 5120), (2, 9000), (1, 20000), (4, 17001)])
def test_norm_behind_a_part_and_layer_norm(n, c, center):
    ops = _ops()
    torch.manual_seed(n + c)
    y, stream, w, b = torch.randn(n, c, device=DEV) + 3.0, torch.randn(n, c, device=DEV), torch.randn(c, device=DEV), torch.randn(c, device=DEV)
    for bias in (None, b):
        for copy_dtype in (None, torch.float32, torch.bfloat16):
            s1, s2 = stream.clone(), stream.clone()
            got = ops.post_norm_add(s1, y, w, 1e-3, bias=bias, copy_dtype=copy_dtype, center=center)
            plain_ops.post_norm_add(s2, y, w, 1e-3, bias=bias, center=center)
            close(s1, s2, 2e-6, "stream")
            assert (got is None) == (copy_dtype is None) and (got is None or torch.equal(got, s1.to(copy_dtype)))
    rows = torch.tensor([n - 1, 0], dtype=torch.int32, device=DEV)
    for delta in (None, stream):
        for which in (None, rows):
            x1, x2 = y.clone(), y.clone()
            got = ops.layer_norm(x1, w, 1e-5, delta=delta, alpha=0.7, rows=which, center=center)
            close(got, plain_ops.layer_norm(x2, w, 1e-5, delta=delta, alpha=0.7, rows=which, center=center), 2e-6, "layer norm")
            close(x1, x2, 1e-6, "rows in front of the norm")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [40, 33, 2048])
def test_embedding_with_positions(hidden, dtype):
    ops = _ops()
    torch.manual_seed(hidden)
    table, pos = torch.randn(50, hidden, device=DEV).to(dtype), torch.randn(30, hidden, device=DEV).to(dtype)
    ids = torch.tensor([0, 49, 7, 7], dtype=torch.int32, device=DEV)
    at = torch.tensor([29, 0, 3, 4], dtype=torch.int32, device=DEV)
    got, copy = ops.embed_positions(ids, table, at, pos, 2.5, copy_dtype=torch.bfloat16)
    want, _ = plain_ops.embed_positions(ids, table, at, pos, 2.5)
    close(got, want, 1e-6, "rows")
    assert torch.equal(copy, got.bfloat16())
    assert ops.embed_positions(ids, table, at, pos)[1] is None


@pytest.mark.parametrize("counts", [[1, 2, 1], [40, 1, 7]])
@pytest.mark.parametrize("channels,taps", [(10, 3), (64, 4), (36, 1), (20, 9)])
def test_convolution_with_silu_behind_it(channels, taps, counts):
    ops, ctx = _ops(), batch(counts)
    torch.manual_seed(channels)
    u, w = torch.randn(ctx.num_tokens, channels + 4, device=DEV), torch.randn(channels, taps, device=DEV)
    states = torch.randn(4, taps - 1, channels, device=DEV) if taps > 1 else None
    slots = torch.tensor([3, 0, 2], dtype=torch.int32, device=DEV)
    s1, s2 = (None, None) if states is None else (states.clone(), states.clone())
    got = ops.short_conv(u, w, s1, slots, ctx, channels=channels, activation="silu")
    close(got, plain_ops.short_conv(u, w, s2, slots, ctx, channels=channels, activation="silu"), 1e-5, "rows")
    if states is not None:
        close(s1, s2, 1e-7, "states")


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("inter", [28, 17, 1024])
def test_gated_activation_with_gelu(inter, dtype, tol):
    ops = _ops()
    torch.manual_seed(inter)
    x, b = (torch.randn(9, 2 * inter, device=DEV) * 2).to(dtype), torch.randn(2 * inter, device=DEV).to(dtype)
    for bias in (None, b):
        close(ops.swiglu(x, bias, "gelu_tanh").float(), plain_ops.swiglu(x, bias, "gelu_tanh").float(), tol, "gelu")
        close(ops.swiglu(x, bias).float(), plain_ops.swiglu(x, bias).float(), tol, "silu")


@pytest.mark.parametrize("cols", [97, 640])
def test_cap_on_logits(cols):
    ops = _ops()
    z = torch.randn(5, cols, device=DEV) * 40
    want = plain_ops.unary(z, "softcap", 12.0)
    close(ops.unary(z, "softcap", 12.0, inplace=True), want, 1e-6, "cap")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [3, 70])
@pytest.mark.parametrize("experts,top,groups", [(16, 4, (4, 2)), (6, 2, (3, 1)), (4, 1, (4, 1)), (128, 8, (8, 4)), (10, 3, None), (2, 2, (1, 1)), (96, 6, (48, 5)), (7, 3, (1, 1))])
def test_router_with_sigmoid_scores_and_groups(experts, top, groups, n, dtype):
    ops = _ops()
    torch.manual_seed(experts + n)
    x, w = torch.randn(n, 80, device=DEV).to(dtype), torch.randn(experts, 80, device=DEV) * 0.3
    # choice scores that are negative for some experts and for all
    for correction in (torch.randn(experts, device=DEV), torch.randn(experts, device=DEV) - 5.0, None):
        got = ops.route(x, w, correction, experts, top, 2.5, True, False, shared_one=True, scores="sigmoid", groups=groups)
        want = plain_ops.route(x, w, correction, experts, top, 2.5, True, False, shared_one=True, scores="sigmoid", groups=groups)
        assert got.shape == want.shape == (n, experts + 1)
        same = ((got != 0) == (want != 0)).all(dim=1)
        assert int((~same).sum()) <= (1 if correction is not None else 2)  # two scores almost equal
        close(got[same], want[same], 1e-5, "weights")


def test_router_takes_the_lowest_index_among_equals():
    ops = _ops()
    x, w = torch.ones(2, 8, device=DEV), torch.zeros(8, 8, device=DEV)
    got = ops.route(x, w, torch.zeros(8, device=DEV), 8, 2, 1.0, True, False, scores="sigmoid", groups=(4, 2))
    assert torch.allclose(got, torch.tensor([[0.5, 0.5, 0, 0, 0, 0, 0, 0]] * 2, device=DEV))
    correction = torch.tensor([0, 0, 1, 0, 0, 1, 0, 0], dtype=torch.float32, device=DEV)
    got = ops.route(x, w, correction, 8, 3, 1.0, True, False, scores="sigmoid", groups=(4, 2))
    assert got[0].nonzero().flatten().tolist() == [2, 3, 5]

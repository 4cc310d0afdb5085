"""The kernels that the Pefedra design added or widened against their plain statements (tests/plain_ops.py) at odd sizes: softmax
attention with two score maps a head, with values that turn back and with a gate a head (both attention kernels); the heads'
preparation with norms over whole projections, two keys a value head and rotated values; the two norms with the token shift
through its state slots; gelu in its erf form behind a product.  And attention inputs built so that one key decides the result,
just inside and just outside the window."""

from __future__ import annotations

import itertools
from types import SimpleNamespace

import pytest
import torch

import plain_ops
from test_kafepel_kernels_gpu import DEV, _ops, close, paged_batch

pytestmark = pytest.mark.gpu

# heads, kv heads, key lanes (of a map), value lanes, page size
SHAPES = [(8, 2, 16, 48, 16), (3, 1, 10, 6, 8), (6, 2, 48, 96, 16), (4, 4, 128, 128, 4), (1, 1, 2, 2, 1), (5, 5, 7, 4, 3), (4, 2, 64, 32, 16),
          (12, 4, 16, 256, 8), (16, 1, 32, 64, 16), (2, 2, 64, 128, 16), (2, 1, 112, 144, 8), (2, 1, 288, 16, 8),
          (6, 2, 64, 64, 32), (4, 1, 64, 128, 8), (4, 2, 128, 128, 16)]


def few_rows(ctx, rows, longest):
    return SimpleNamespace(positions=ctx.positions[rows].contiguous(), token_request=ctx.token_request[rows].contiguous(), max_context_len=longest,
                           max_query_len=1, num_requests=len(rows), num_tokens=len(rows), context_lens=ctx.context_lens,
                           cu_tokens=torch.arange(len(rows) + 1, dtype=torch.int32, device=DEV), host_cu_tokens=list(range(len(rows) + 1)))


def variants(ops, H, V, N, gate):
    diff = ops.DifferentialMaps(0.7, 1e-5, 0.6)
    turn = torch.rand(N, V // 2, device=DEV) * 6.0
    turn = torch.stack((turn.cos(), turn.sin()), dim=-1).contiguous()
    lanes = torch.randn(N, H * V + 3, device=DEV)[:, 1 : 1 + H * V]
    return [
        ("two maps, a window", dict(differential=diff, window=33)),
        ("two maps, all keys", dict(differential=diff)),
        ("two maps, a window of one", dict(differential=diff, window=1)),
        ("two maps, values that turn back, a gate a head, a cap", dict(differential=diff, window=70, turn=turn, gate=gate, gate_per_head=True, softcap=2.0)),
        ("two maps and a gate a lane", dict(differential=diff, window=70, gate=lanes)),
        ("values that turn back, a gate a head", dict(window=64, turn=turn, gate=gate, gate_per_head=True)),
        ("values that turn back, neighbouring lanes", dict(turn=turn, turn_neighbours=True)),
        ("values that turn back, a gate a lane", dict(window=9, turn=turn, gate=lanes)),
        ("a gate a head", dict(window=100, gate=gate, gate_per_head=True)),
    ]


def use_kernels(monkeypatch, ops, way: str) -> None:
    """``tcgen05``: as the engine chooses (requests of 128 tokens and more of some sizes on tcgen05); ``mma``: the row kernel also
    there; ``general``: the kernel for any sizes also where a tensor-core kernel would run."""
    monkeypatch.setattr(ops, "_FORCE_GENERIC_ATTENTION", way == "general")
    monkeypatch.setattr(ops, "_TC_ATTENTION_ENABLED", way == "tcgen05")


@pytest.mark.parametrize("dtype,tol,way", [(torch.float32, 2e-5, "general"), (torch.bfloat16, 2e-2, "general"), (torch.bfloat16, 2e-2, "mma"),
                                           (torch.bfloat16, 2e-2, "tcgen05")])
@pytest.mark.parametrize("H,KV,D,V,page_size", SHAPES)
def test_maps_turns_and_gates_against_plain(H, KV, D, V, page_size, dtype, tol, way, monkeypatch):
    """Long and short requests in one step.  The result goes into rows with a pitch."""
    ops = _ops()
    use_kernels(monkeypatch, ops, way)
    torch.manual_seed(H * 100 + D + 2)
    ctx, table, slots, pages = paged_batch([37, 1, 340, 1300, 550], [5, 1, 200, 2, 131], page_size)
    N = ctx.num_tokens
    gate = torch.randn(N, H + 4, device=DEV)[:, 2 : 2 + H]
    rows = [4, 5, 205, 207]
    few = few_rows(ctx, rows, 1300)
    few.context_lens = ctx.context_lens[:4].contiguous()
    for what, more in variants(ops, H, V, N, gate):
        maps = 2 if "differential" in more else 1
        if maps * D > 640:
            continue
        pool = (torch.randn(pages, 2, KV, page_size, max(maps * D, V), device=DEV) * 0.7).to(dtype)
        q = torch.randn(N, H * maps * D, device=DEV).to(dtype)
        common = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=0.3)
        full = plain_ops.paged_softmax_attention(q, pool, table, ctx, **common, **more)
        wide = torch.zeros(N, H * V + 16, device=DEV, dtype=dtype)
        ops.paged_softmax_attention(q, pool, table, ctx, **common, **more, out=wide[:, 8 : 8 + H * V])
        # the difference of two maps is normed: where the maps nearly cancel, rounding before the norm shows behind it
        close(wide[:, 8 : 8 + H * V], full, tol * (3 if maps == 2 else 1), what)
        assert not wide[:, :8].any() and not wide[:, 8 + H * V :].any(), f"{what}: written beside the rows"
        # the same rows as single tokens of a small step (long contexts are cut over several CTAs)
        part = {k: (v[rows].contiguous() if k in ("turn", "gate") else v) for k, v in more.items()}
        close(ops.paged_softmax_attention(q[rows].contiguous(), pool, table, few, **common, **part), full[rows], tol * (3 if maps == 2 else 1), what + ", single tokens")


@pytest.mark.parametrize("dtype,way,D", [(torch.float32, "general", 32), (torch.bfloat16, "general", 32), (torch.bfloat16, "mma", 32), (torch.bfloat16, "tcgen05", 64)])
@pytest.mark.parametrize("news", [[600, 1, 1], [1, 1, 1], [64, 2, 1], [300, 131, 3]])
def test_one_key_at_the_window_decides_in_each_map(news, dtype, way, D, monkeypatch):
    """Keys are built from the three base-9 digits of their position (a third of a unit vector per digit), so that a query 66 times
    key j scores 66 on key j and at most 44 on any other visible key.  The first map asks for one key and the second for another:
    with a difference weight of 1/2 and no norm to speak of (eps far above the rows' size, the scale its root) the result is the
    first key's value row less half the second's.  Asked for: the key just inside and just outside a window of 70, keys at page
    borders and the query's own, in either map."""
    ops = _ops()
    use_kernels(monkeypatch, ops, way)
    H, KV, V, page_size, W = 4, 2, (64 if D == 64 else 16), 8, 70
    lens = [600, 523, 300]
    ctx, table, slots, pages = paged_batch(lens, news, page_size, seed=3)
    pool = torch.zeros(pages, 2, KV, page_size, 2 * D, device=DEV, dtype=dtype)
    j = torch.arange(max(lens))
    code = torch.zeros(max(lens), D)
    for digit in range(3):
        code[j, 9 * digit + (j // 9 ** digit) % 9] = 3 ** -0.5
    vals = {r: torch.randn(n, KV, V) for r, n in enumerate(lens)}
    host_table = table.cpu()
    for r, n in enumerate(lens):
        for jj in range(n):
            page, off = int(host_table[r, jj // page_size]), jj % page_size
            pool[page, 0, :, off] = torch.cat((code[jj], code[jj])).to(dtype)
            pool[page, 1, :, off, :V] = vals[r][jj].to(dtype)
    positions, owner = ctx.positions.cpu().tolist(), ctx.token_request.cpu().tolist()
    diff = ops.DifferentialMaps(0.5, 1e8, 1e4)
    common = dict(num_heads=H, num_kv_heads=KV, key_dim=D, value_dim=V, scale=1.0, window=W, differential=diff)
    edge, own = (lambda p: max(0, p - W + 1)), (lambda p: p)
    beyond = lambda p: max(0, p - W)  # noqa: E731  (outside the window, for p >= W)
    border = lambda p: max(0, p - p % page_size - 1) if p - (p - p % page_size - 1) < W else p  # noqa: E731  (the last key of the page in front)
    tol = 2e-4 if dtype == torch.float32 else 4e-2
    for what, first, second in (("edge and own", edge, own), ("own and edge", own, edge), ("page border and edge", border, edge), ("beyond and own", beyond, own),
                                ("own and beyond", own, beyond)):
        asked = [[first(p) for p in positions], [second(p) for p in positions]]
        q = torch.stack([torch.cat((code[a] * 66.0, code[b] * 66.0)) for a, b in zip(*asked)]).repeat(1, H).to(DEV).to(dtype)
        out = ops.paged_softmax_attention(q, pool, table, ctx, **common).float().cpu()
        reference = plain_ops.paged_softmax_attention(q, pool, table, ctx, **common).float().cpu()
        assert float((out - reference).abs().max()) <= tol, what
        for i, p in enumerate(positions):
            a, b = asked[0][i], asked[1][i]
            row = lambda t: vals[owner[i]][t].repeat_interleave(H // KV, dim=0).reshape(-1).to(dtype).float()  # noqa: E731,B023
            want = row(a) - 0.5 * row(b)
            if p - a < W and p - b < W:
                assert float((out[i] - want).abs().max()) <= tol, f"{what}: position {p} does not get keys {a} and {b}"
            elif float((reference[i] - want).abs().max()) > 10 * tol:
                assert float((out[i] - want).abs().max()) > 5 * tol, f"{what}: position {p} sees a key beyond its window"


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("H,KV,D,V,page_size", SHAPES)
def test_head_prepare_whole_norms_two_keys_and_rotated_values(H, KV, D, V, page_size, dtype, tol):
    ops = _ops()
    torch.manual_seed(H * 100 + D + 3)
    ctx, table, slots, pages = paged_batch([37, 1, 200, 530], [5, 1, 200, 2], page_size)
    N = ctx.num_tokens
    rot = D // 2 * 2 if D < 64 else D // 4 * 2
    freq, vfreq = torch.rand(rot // 2, device=DEV), torch.rand(V // 2, device=DEV)
    for maps in (1, 2):
        keys = KV * maps
        cols = (H * maps + keys) * D + KV * V
        proj, bias = torch.randn(N, cols + 8, device=DEV), torch.randn(cols, device=DEV)
        qw, kw = torch.randn(H * maps * D, device=DEV), torch.randn(keys * D, device=DEV)
        for what, more in (
            ("whole norms and bias", dict(bias=bias, q_weight=qw, k_weight=kw, eps=1e-5, norm_whole=True, freq=freq)),
            ("rotated values", dict(bias=bias, freq=freq, value_freq=vfreq)),
            ("rotated values, neighbouring lanes, whole norms", dict(q_weight=qw, k_weight=kw, eps=1e-3, norm_whole=True, value_freq=vfreq, interleaved=True)),
            ("bias and rotation alone", dict(bias=bias, freq=freq)),
        ):
            p1 = (torch.randn(pages, 2, KV, page_size, max(maps * D, V), device=DEV) * 0.5).to(dtype)
            p2 = p1.clone()
            t1, t2 = (torch.zeros(N, V // 2, 2, device=DEV) for _ in range(2)) if "value_freq" in more else (None, None)
            kwargs = dict(heads=H * maps, kv_heads=keys, dim=D, value_dim=V, slot_map=slots, out_dtype=dtype, maps=maps, **more)
            q1 = ops.head_prepare(proj, ctx.positions, pool=p1, turn_out=t1, **kwargs)
            q2 = plain_ops.head_prepare(proj, ctx.positions, pool=p2, turn_out=t2, **kwargs)
            close(q1, q2, tol, f"{what}, {maps} maps: queries")
            close(p1, p2, tol, f"{what}, {maps} maps: keys and values in their pages")
            if t1 is not None:
                close(t1, t2, 2e-4, what + ": cosines and sines")


def ctx_of(counts):
    cu = torch.tensor([0] + list(itertools.accumulate(counts)), dtype=torch.int32, device=DEV)
    owner = torch.repeat_interleave(torch.arange(len(counts), dtype=torch.int32), torch.tensor(counts)).to(DEV)
    return SimpleNamespace(cu_tokens=cu, token_request=owner, num_requests=len(counts), max_query_len=max(counts))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("W", [1, 7, 40, 64, 130, 1024, 1028, 2048, 3000, 4100, 8192, 8200])
def test_shift_norm_against_plain_and_across_ways_of_cutting(W, dtype, tol):
    """Unequal requests in one step against the plain statement; then the same tokens in portions down to one token through the
    state slots: bit-equal results whatever the cut, and slots that hold the last unshifted row."""
    ops = _ops()
    torch.manual_seed(W)
    lens = [70, 1, 19, 33]
    N = sum(lens)
    x = torch.randn(N, W, device=DEV) * 3
    w1, w2, shift = torch.randn(W, device=DEV), torch.randn(W, device=DEV), torch.rand(W, device=DEV) * 1.4 - 0.2
    slots = torch.tensor([2, 0, 5, 3], dtype=torch.int32, device=DEV)
    s1 = torch.zeros(6, W, device=DEV)
    s2 = s1.clone()
    whole = ops.shift_norm(x, w1, 1e-5, w2=w2, shift=shift, states=s1, ctx=ctx_of(lens), state_slots=slots, out_dtype=dtype)
    ref = plain_ops.shift_norm(x, w1, 1e-5, w2=w2, shift=shift, states=s2, ctx=ctx_of(lens), state_slots=slots, out_dtype=dtype)
    close(whole[0], ref[0], tol, "shifted rows")
    close(whole[1], ref[1], tol, "the second norm")
    close(s1, s2, 2e-6, "the slots")
    plain, none = ops.shift_norm(x, w1, 1e-5, out_dtype=dtype)
    assert none is None
    close(plain, ops.rmsnorm(x.clone(), w1, 1e-5, out_dtype=dtype), tol, "without a shift and a second norm: an RMS norm")
    s3, at, starts = torch.zeros_like(s1), 0, [0, 70, 71, 90]
    got = [torch.empty_like(whole[0]), torch.empty_like(whole[1])]
    for step, n in enumerate((1, 2, 5, 1, 40, 21)):
        rows, counts, sl = list(range(at, at + n)), [n], [2]
        if step < 3:
            rows += list(range(starts[step + 1], starts[step + 1] + lens[step + 1]))
            counts.append(lens[step + 1])
            sl.append(int(slots[step + 1]))
        part = ops.shift_norm(x[rows].contiguous(), w1, 1e-5, w2=w2, shift=shift, states=s3, ctx=ctx_of(counts),
                              state_slots=torch.tensor(sl, dtype=torch.int32, device=DEV), out_dtype=dtype)
        for g, p in zip(got, part):
            g[rows] = p
        at += n
    assert torch.equal(got[0], whole[0]) and torch.equal(got[1], whole[1]), "the rows depend on how the tokens were cut"
    assert torch.equal(s3, s1), "the slots depend on how the tokens were cut"


def test_shift_norm_of_a_long_step():
    """So many tokens that a CTA walks several, across the borders of requests."""
    ops = _ops()
    torch.manual_seed(1)
    lens = [1500, 3, 1, 2100, 700, 1, 1]
    N, W = sum(lens), 96
    x = torch.randn(N, W, device=DEV)
    w1, w2, shift = torch.randn(W, device=DEV), torch.randn(W, device=DEV), torch.rand(W, device=DEV)
    slots = torch.tensor([6, 1, 0, 2, 5, 3, 4], dtype=torch.int32, device=DEV)
    s1 = torch.randn(7, W, device=DEV)
    s2 = s1.clone()
    a = ops.shift_norm(x, w1, 1e-6, w2=w2, shift=shift, states=s1, ctx=ctx_of(lens), state_slots=slots)
    b = plain_ops.shift_norm(x, w1, 1e-6, w2=w2, shift=shift, states=s2, ctx=ctx_of(lens), state_slots=slots)
    close(a[0], b[0], 2e-6, "shifted rows")
    close(a[1], b[1], 2e-6, "the second norm")
    close(s1, s2, 2e-6, "the slots")


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("N,K,F", [(1, 64, 40), (8, 128, 256), (16, 192, 33), (5, 40, 24), (130, 128, 96), (3, 2048, 512)])
def test_gelu_behind_a_product(N, K, F, dtype, tol):
    """The erf form, alone and as the end of a product, into rows with a pitch; far from the tanh form's values nowhere, but
    further from them than the tolerance somewhere in 32-bit."""
    ops = _ops()
    torch.manual_seed(N + K)
    x, w = torch.randn(N, K, device=DEV).to(dtype), (torch.randn(F, K, device=DEV) * K ** -0.5 * 2).to(dtype)
    wide = torch.zeros(N, F + 24, device=DEV, dtype=dtype)
    ops.linear_act(x, w, "gelu", out=wide[:, 16 : 16 + F])
    z = x.float() @ w.float().t()
    close(wide[:, 16 : 16 + F], 0.5 * z * (1 + torch.erf(z * 0.5**0.5)), tol, "product and gelu")
    assert not wide[:, :16].any() and not wide[:, 16 + F :].any()
    close(ops.linear_act(x, w, "gelu"), plain_ops.linear_act(x, w, "gelu"), tol, "without a place to go")
    if dtype == torch.float32 and N * F > 1000:
        line = torch.linspace(-6, 6, 4096, device=DEV)[None]
        exact, other = ops.unary(line, "gelu"), ops.unary(line, "gelu_tanh")
        assert float((exact - 0.5 * line * (1 + torch.erf(line * 0.5**0.5))).abs().max()) < 2e-6 < 1e-4 < float((exact - other).abs().max())

"""Kernels of linear recurrences, paired attention, grouped routing and normed polynomials against the definitions on the CPU."""

import dataclasses

import pebodra_oracle as O
import pytest
import torch

from slime_b200.ops import grouped, linear_scan, stream
from slime_b200.ops import window_attention as wa

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.bfloat16, torch.float32]


def _close(got, want, tol):
    err = float((got.float().cpu() - want.float().cpu()).abs().max())
    assert err < tol * max(1.0, float(want.float().abs().max())), err


def _cut(x, lo, hi, names):
    return dataclasses.replace(x, **{n: getattr(x, n)[lo:hi] for n in names})


def _columns(g, T, widths, dtype):
    """Column ranges of one matrix, each starting at a multiple of 8."""
    up8 = lambda n: -(-n // 8) * 8  # noqa: E731
    x, at, out = torch.randn(T, sum(up8(w) for w in widths), generator=g).to(dtype), 0, []
    for w in widths:
        out.append(slice(at, at + w))
        at += up8(w)
    return lambda dev, dt: [x.to(dev, dt)[:, s] for s in out]


# heads, groups, state, value width, taps, normed parts
SPACES = [(4, 2, 32, 64, 4, 2), (6, 1, 64, 32, 4, 3), (2, 2, 128, 64, 4, 1), (3, 1, 96, 48, 3, 3), (5, 5, 20, 72, 2, 1), (1, 1, 9, 7, 1, 7), (4, 2, 40, 16, 6, 4),
          (2, 1, 200, 160, 4, 2), (8, 4, 128, 128, 4, 1), (2, 1, 300, 20, 9, 1), (3, 3, 16, 6, 4, 2)]  # fmt: skip


def _space(shape, T, dtype):
    H, G, N, DV, taps, parts = shape
    g = torch.Generator().manual_seed(sum(shape))
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    cols, ch = _columns(g, T, [H * DV, H * DV, G * N, G * N, H], dtype), H * DV + 2 * G * N
    conv, conv_b, norm = ((r(*s) * 0.5).to(dtype) for s in ((ch, taps), (ch,), (H * DV,)))
    A, bias, skip = r(H) - 1, r(H) - 2, r(H)

    def on(dev, dt=None):
        dt = dt or dtype
        return linear_scan.StateSpace(*cols(dev, dt), conv.to(dev, dt), conv_b.to(dev, dt), A.to(dev), bias.to(dev), skip.to(dev), norm.to(dev, dt), parts, 1e-3)

    def state(dev, dt, fill):
        new = lambda *s: torch.full(s, fill, device=dev)  # noqa: E731
        return linear_scan.SlotState(new(3, H, N, DV), new(3, taps, ch).to(dt))

    return on, state, ("z", "x", "B", "C", "dt")


# heads, key width, value width
MEMORIES = [(4, 32, 64), (3, 20, 28), (2, 128, 96), (8, 256, 512), (1, 9, 7), (2, 300, 40), (5, 64, 16), (2, 6, 130)]


def _memory(shape, T, dtype):
    H, D, DV = shape
    g = torch.Generator().manual_seed(sum(shape))
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    cols = _columns(g, T, [H * D, H * D, H * DV, H, H, H * DV], dtype)
    i_b, f_b, norm = r(H) * 2, r(H) + 3, (r(H * DV) * 0.5).to(dtype)

    def on(dev, dt=None):
        dt = dt or dtype
        return linear_scan.MatrixMemory(*cols(dev, dt), i_b.to(dev), f_b.to(dev), norm.to(dev, dt), 9.0, 1e-3)

    def state(dev, dt, fill):
        new = lambda *s: torch.full(s, fill, device=dev)  # noqa: E731
        return linear_scan.SlotState(new(3, H, D, DV), None, new(3, H, D), new(3, H, 2))

    return on, state, ("q", "k", "v", "i", "f", "z")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make,shape", [(_space, s) for s in SPACES] + [(_memory, s) for s in MEMORIES])
def test_portions_and_steps(kernels, make, shape, dtype):
    """Portions, then single tokens, in a slot that held something else, against one pass of the definition; other slots stay."""
    T, tol = 150, 3e-2 if dtype == torch.bfloat16 else 2e-4
    on, state, names = make(shape, T, dtype)
    cpu, gpu = on("cpu", torch.float32), on(DEV)
    want_state, got_state = state("cpu", torch.float32, 0.0), state(DEV, dtype, 7.0)
    seg = lambda at, n, dev: wa.ExtendBatch.build([[0]], [at], [n], 256, dev, state_slots=[1])  # noqa: E731
    want = cpu.extend(want_state, seg(0, T, "cpu"))
    got, at, one = [], 0, torch.ones(1, dtype=torch.int32, device=DEV)
    for n in (70, 1, 2, 17, 3, 37):
        got.append(_cut(gpu, at, at + n, names).extend(got_state, seg(at, n, DEV)))
        at += n
    for t in range(at, T):
        got.append(_cut(gpu, t, t + 1, names).step(got_state, one, one, one * t))
    _close(torch.cat(got), want, tol)
    for n in ("state", "ring", "norm"):
        a, b = getattr(got_state, n), getattr(want_state, n)
        if a is not None and not (n == "ring" and a.shape[1] == 1):
            rows = [(T - 1 - i) % a.shape[1] for i in range(a.shape[1] - 1)] if n == "ring" else slice(None)
            _close(a[1][rows], b[1][rows], tol)
            assert (a[[0, 2]].float() == 7).all()
    if got_state.top is not None:
        _close(got_state.top[1, :, T % 2], want_state.top[1, :, T % 2], tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make,shape", [(_space, SPACES[0]), (_space, SPACES[4]), (_memory, MEMORIES[0]), (_memory, MEMORIES[1])])
def test_batches_and_idle_rows(kernels, make, shape, dtype):
    """Requests of unequal length in one pass, one of them continued; a step with idle rows in any order of slots."""
    T, tol = 120, 3e-2 if dtype == torch.bfloat16 else 2e-4
    on, state, names = make(shape, T, dtype)
    cpu, gpu = on("cpu", torch.float32), on(DEV)
    a, b = state("cpu", torch.float32, 0.0), state(DEV, dtype, 0.0)
    for s, x, dev in ((a, cpu, "cpu"), (b, gpu, DEV)):
        s.first = _cut(x, 0, 40, names).extend(s, wa.ExtendBatch.build([[0]], [0], [40], 256, dev, state_slots=[2]))
        batch = wa.ExtendBatch.build([[0]] * 3, [0, 40, 0], [1, 33, 43], 256, dev, state_slots=[0, 2, 1])
        s.second = _cut(x, 40, 117, names).extend(s, batch)
        i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=dev)  # noqa: E731, B023
        s.third = _cut(x, 117, 120, names).step(s, i32(2, 1, 0), i32(1, 0, 1), i32(73, 43, 1))
    for n in ("first", "second", "third"):
        _close(getattr(b, n)[[0, 2]] if n == "third" else getattr(b, n), getattr(a, n)[[0, 2]] if n == "third" else getattr(a, n), tol)
    _close(b.state, a.state, tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make,shape", [(_space, (44, 4, 100, 56, 4, 4)), (_space, (40, 1, 128, 64, 3, 1)), (_memory, (10, 200, 300)), (_memory, (50, 128, 20))])
def test_many_heads_and_requests(kernels, make, shape, dtype):
    """Enough work to fill the machine: the form of the scan with more columns per lane."""
    counts, tol = [31, 8, 1, 40], 3e-2 if dtype == torch.bfloat16 else 2e-4
    T = sum(counts)
    on, state, names = make(shape, T, dtype)
    res = []
    for x, dev, dt in ((on("cpu", torch.float32), "cpu", torch.float32), (on(DEV), DEV, dtype)):
        s = state(dev, dt, 0.0)
        s = linear_scan.SlotState(*(None if t is None else torch.cat([t, t]) for t in (s.state, s.ring, s.norm, s.top)))
        batch = wa.ExtendBatch.build([[0]] * 4, [0] * 4, counts, 256, dev, state_slots=[4, 0, 2, 5])
        res.append((x.extend(s, batch), s.state, s.norm if s.norm is not None else s.state))
    for a, b in zip(*res):
        _close(b, a, tol)


@pytest.mark.parametrize("make,shape", [(_space, (6, 2, 100, 40, 4, 2)), (_space, (4, 4, 16, 20, 2, 1)), (_memory, (4, 40, 24)), (_memory, (3, 180, 70))])
def test_decays_of_any_strength(kernels, make, shape):
    """Heads that forget everything at once, heads that forget slowly, and a change of mind in the middle of a prompt."""
    T, H = 90, shape[0]
    on, state, names = make(shape, T, torch.float32)
    res = []
    for dev in ("cpu", DEV):
        x = on(dev)
        strength = torch.linspace(-3.0, 6.0, H, device=dev)
        if make is _space:
            x.A_log[:] = strength
            x.dt[40:60] = 8.0
        else:
            x.f_b[:] = 4.0 - 3 * strength
            x.i[40:43] = 30.0  # an input that takes over
        s = state(dev, torch.float32, 0.0)
        out = [_cut(x, a, b, names).extend(s, wa.ExtendBatch.build([[0]], [a], [b - a], 256, dev, state_slots=[1])) for a, b in ((0, 37), (37, 90))]
        res.append((torch.cat(out), s.state[1]))
    for a, b in zip(*res):
        assert torch.isfinite(a).all()
        _close(b, a, 2e-4)


def test_a_long_scan_keeps_a_far_token(kernels):
    """3000 tokens with decays near one: the first one still shows, in portions and in one pass alike."""
    H, D, DV, T = 2, 64, 64, 3000
    on, state, names = _memory((H, D, DV), T, torch.float32)
    x = on(DEV)
    x.f[:], x.i[:] = 9.0, 0.0
    seg = lambda at, n: wa.ExtendBatch.build([[0]], [at], [n], 4096, DEV, state_slots=[0])  # noqa: E731
    s1, s2 = state(DEV, None, 0.0), state(DEV, None, 0.0)
    whole = x.extend(s1, seg(0, T))
    parts = torch.cat([_cut(x, a, b, names).extend(s2, seg(a, b - a)) for a, b in ((0, 1), (1, 1501), (1501, T))])
    assert float((whole - parts).abs().max()) < 1e-4
    v0 = x.v[0].clone()
    x.v[0] *= -40
    assert float((x.extend(state(DEV, None, 0.0), seg(0, T))[-1] - whole[-1]).abs().max()) > 1e-3
    x.v[0] = v0
    S, n, m = torch.zeros(H, D, DV, dtype=torch.float64), torch.zeros(H, D, dtype=torch.float64), torch.zeros(H, dtype=torch.float64)
    q, k, v = (t.double().cpu().view(T, H, -1) for t in (x.q * D**-0.5, x.k, x.v))
    soft = lambda z: 9.0 * torch.tanh(z.double().cpu() / 9.0)  # noqa: E731
    i, g = soft(x.i + x.i_b), O.log_sigmoid(soft(x.f + x.f_b))
    for t in range(T):
        new = torch.maximum(g[t] + m, i[t])
        f, w, m = torch.exp(g[t] + m - new), torch.exp(i[t] - new), new
        S = f[:, None, None] * S + w[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = f[:, None] * n + w[:, None] * k[t]
    _close(s1.state[0], S, 1e-4)
    _close(s1.norm[0], n, 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,P,W", [(5, 3, 40), (70, 2, 512), (3, 1, 1200), (9, 4, 7), (2, 2, 5000), (1, 1, 4100)])
def test_part_gate(kernels, T, P, W, dtype):
    g = torch.Generator().manual_seed(W)
    o, z, w = torch.randn(T, P * W, generator=g), torch.randn(T, P * W, generator=g).to(dtype), torch.randn(P * W, generator=g).to(dtype)
    den = torch.rand(T, P, generator=g) + 0.5
    tol = 2e-2 if dtype == torch.bfloat16 else 1e-5
    for act, first, d in (("silu", True, None), ("sigmoid", False, den), ("silu", False, None), ("sigmoid", True, den)):
        want = linear_scan.part_gate(o, z.float(), w.float(), P, act, 0.01, gate_first=first, den=d, scale=0.7)
        out = torch.zeros(T, P * W + 8, dtype=dtype, device=DEV)
        got = linear_scan.part_gate(o.to(DEV), z.to(DEV), w.to(DEV), P, act, 0.01, gate_first=first, den=None if d is None else d.to(DEV), scale=0.7,
                                    out=out[:, : P * W])  # fmt: skip
        _close(got, want, tol)
        assert not out[:, P * W :].any()


def _paged(lengths, ps, dtype, g, *shapes):
    count = [-(-n // ps) for n in lengths]
    order = torch.randperm(sum(count) + 2, generator=g).tolist()
    pages = [[order.pop() for _ in range(c)] for c in count]
    caches = []
    for s in shapes:
        c = torch.full(((sum(count) + 2) * ps, *s), float("nan"))
        for p, n in zip(pages, lengths):
            i = torch.arange(n)
            c[torch.tensor(p)[i // ps] * ps + i % ps] = torch.randn(n, *s, generator=g).to(dtype).float()
        caches.append(c)
    return pages, caches


# heads, kv heads, width of a half, value width
PAIRS = [(4, 2, 32, 64), (16, 8, 64, 128), (8, 1, 64, 64), (6, 2, 24, 40), (3, 3, 16, 128), (2, 1, 48, 16), (4, 1, 10, 13), (2, 2, 80, 160), (40, 1, 16, 32)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 40, 129, None])
@pytest.mark.parametrize("shape", PAIRS)
def test_difference_of_two_attentions(kernels, shape, window, dtype):
    H, G, D, DV = shape
    g = torch.Generator().manual_seed(H + D)
    lengths, starts, ps = [300, 129, 1, 77], [0, 100, 0, 75], 16
    pages, (kc, vc) = _paged(lengths, ps, dtype, g, (G, 2 * D), (G, DV))
    counts = [n - s for n, s in zip(lengths, starts)]
    T = sum(counts)
    q = torch.zeros(T, H, 2, 2, D)
    q[:, :, 0, 0], q[:, :, 1, 1] = (torch.randn(T, H, D, generator=g).to(dtype).float() for _ in range(2))
    q = q.view(T, 2 * H, 2 * D)
    weight, form = torch.tensor([0.45]), dict(scale=1.5 * D**-0.5, window=window)
    build = lambda dev: wa.ExtendBatch.build(pages, starts, counts, ps, dev)  # noqa: E731
    want = wa.window_extend(q, kc, vc, build("cpu"), **form, pair=wa.Pair(weight, 0.6, 1e-3))
    pair = wa.Pair(weight.to(DEV), 0.6, 1e-3)
    k, v = (c.nan_to_num(0.0).to(DEV, dtype) if dtype == torch.float32 else c.to(DEV, dtype) for c in (kc, vc))
    out = torch.zeros(T, H * DV + 8, dtype=dtype, device=DEV)
    tol = 4e-2 if dtype == torch.bfloat16 else 1e-4
    _close(wa.window_extend(q.to(DEV, dtype), k, v, build(DEV), **form, pair=pair, out=out[:, : H * DV]), want, tol)
    assert not out[:, H * DV :].any()
    last = torch.tensor(lengths, dtype=torch.int32, device=DEV)
    rows = [sum(counts[: i + 1]) - 1 for i in range(len(counts))]
    for most in (512, 8192):  # few and many key ranges
        got = wa.window_decode(q[rows].to(DEV, dtype), k, v, build(DEV).block_table, last, last - 1, ps, **form, max_context=most, pair=pair)
        _close(got, want[rows], tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("own", [True, False])
def test_pairs_of_heads_are_placed(kernels, own, dtype):
    for H, G, D, DV, dims in ((3, 3, 10, 7, 6), (8, 2, 64, 128, 64), (4, 4, 32, 48, 20)):
        T, g = 33, torch.Generator().manual_seed(D)
        x = torch.randn(T, (H + G) * 2 * D + G * DV, generator=g).to(dtype)
        wq, wk = (torch.randn(D, generator=g).to(dtype) for _ in range(2))
        pos, slots = torch.randint(0, 200, (T,), generator=g).int(), torch.randperm(40, generator=g)[:T].int()
        slots[3] = -1
        res = []
        for dev in ("cpu", DEV):
            dt = torch.float32 if dev == "cpu" else dtype
            q, k, v = x.to(dev, dt).split([H * 2 * D, G * 2 * D, G * DV], 1)
            kc, vc = torch.zeros(40, G, 2 * D, dtype=dt, device=dev), torch.zeros(40, G, DV, dtype=dt, device=dev)
            y = stream.place_heads(q, k if own else None, v if own else None, slots.to(dev), kc, vc, q_norm=wq.to(dev, dt), k_norm=wk.to(dev, dt) if own else None,
                                   eps=1e-3, table=stream.rotary_table(200, dims, 30.0, dev), positions=pos.to(dev), interleaved=False, maps=2)  # fmt: skip
            res.append((y, kc, vc))
        for a, b in zip(*res):
            _close(b, a, 2e-2 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("experts,top,groups", [(20, 3, (5, 2)), (128, 8, (8, 4)), (6, 2, (6, 3)), (512, 8, (32, 5)), (9, 2, (3, 1)), (7, 7, (1, 1)), (256, 4, (2, 1))])
def test_router_prefers_good_groups(kernels, experts, top, groups):
    g = torch.Generator().manual_seed(experts)
    z, bias = torch.randn(300, experts, generator=g) * 2, torch.randn(experts, generator=g) * 0.1
    for b, renorm in ((None, False), (bias, True)):
        w, idx = grouped.route_topk(z, top, score="sigmoid", renorm=renorm, bias=b, groups=groups)
        w2, idx2 = grouped.route_topk(z.to(DEV), top, score="sigmoid", renorm=renorm, bias=None if b is None else b.to(DEV), groups=groups)
        assert torch.equal(idx2.cpu(), idx)
        torch.testing.assert_close(w2.cpu(), w, atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_normed_polynomial_and_cap(kernels, dtype):
    g = torch.Generator().manual_seed(2)
    tol = 2e-2 if dtype == torch.bfloat16 else 1e-5
    for T, F in ((3, 37), (70, 392), (5, 9728), (2, 20000), (2, 2051)):
        wide = (torch.randn(T, F + 8, generator=g) * 2).to(dtype)
        z, coef = wide[:, :F], torch.randn(4, generator=g)
        want = stream.poly_norm(z.float(), coef, 1e-3)
        _close(stream.poly_norm(wide.to(DEV)[:, :F], coef.to(DEV), 1e-3), want, tol)
        sums = stream.poly_sums(z.float())
        _close(stream.poly_norm(wide.to(DEV)[:, : F // 2], coef.to(DEV), 1e-3, sums.to(DEV), F), want[:, : F // 2], tol)
    x = torch.randn(5, 1003, generator=g) * 40
    _close(stream.softcap_(x.to(DEV)[:, :1000], 9.0), 9.0 * torch.tanh(x[:, :1000] / 9.0), 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,groups", [(288, 4), (90, 2), (96, 3), (2560, 4), (40, 1), (4096, 64), (77, 77), (8192, 8)])
def test_norms_of_parts_around_the_stream(kernels, H, groups, dtype):
    T, g = 19, torch.Generator().manual_seed(H)
    y, res = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g)
    w, pre = (torch.randn(H, generator=g).to(dtype) for _ in range(2))
    tol = 2e-2 if dtype == torch.bfloat16 else 1e-5
    for p, emit in ((pre, None), (None, dtype), (None, None)):
        want = stream.stream_norm(y, res.clone(), None if p is None else p.float(), 1e-3, post_w=w.float(), groups=groups, emit=None if emit is None else torch.float32)
        got = stream.stream_norm(y.to(DEV), res.to(DEV), None if p is None else p.to(DEV), 1e-3, post_w=w.to(DEV), groups=groups, emit=emit)
        _close(got[1], want[1], 1e-5)
        assert (got[0] is None) == (want[0] is None)
        if got[0] is not None:
            assert got[0].dtype == dtype
            _close(got[0], want[0], tol)

"""Kernels of the gated delta rule, of head preparation and of the pair table against the definitions on the CPU."""

import dataclasses

import pytest
import torch

from slime_b200.ops import delta, stream
from slime_b200.ops import window_attention as wa

pytestmark = pytest.mark.gpu
DEV = "cuda"
# heads, query/key heads, key width, value width, taps
SHAPES = [(4, 2, 32, 64, 4), (6, 6, 64, 32, 4), (2, 1, 128, 128, 4), (3, 3, 96, 48, 3), (5, 1, 20, 72, 2), (1, 1, 9, 7, 1), (4, 2, 40, 16, 6),
          (2, 2, 200, 160, 4), (3, 1, 128, 256, 5), (2, 2, 64, 100, 4), (2, 1, 16, 20, 8), (2, 2, 72, 128, 4)]  # fmt: skip


def _inputs(shape, per_channel, T, dtype, seed=0):
    """Projections as column ranges of one matrix (q, k, v, b; a from another product), gates near one so that old writes last."""
    H, G, D, DV, taps = shape
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    up8 = lambda n: -(-n // 8) * 8  # noqa: E731
    widths = [G * D, G * D, H * DV, H]
    x, at, cols = r(T, sum(up8(w) for w in widths)).to(dtype), 0, []
    for w in widths:
        cols.append(slice(at, at + w))
        at += up8(w)
    a = r(T, up8(H * D if per_channel else H)).to(dtype) - 2
    conv, rate, bias = (r(2 * G * D + H * DV, taps) * 0.6).to(dtype), r(H) * 0.5, r(H * D if per_channel else H) - 2

    def on(dev, dt=None):
        y, b, c = (t.to(dev, dt or dtype) for t in (x, a, conv))
        q, k, v, beta = (y[:, s] for s in cols)
        return delta.DeltaInputs(q, k, v, b[:, : bias.numel()], beta, c, rate.to(dev), bias.to(dev))

    return on


def _cut(x, lo, hi):
    return dataclasses.replace(x, **{n: getattr(x, n)[lo:hi] for n in "qkvab"})


def _close(got, want, tol):
    err = float((got.float().cpu() - want.float().cpu()).abs().max())
    assert err < tol * max(1.0, float(want.float().abs().max())), err


@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES)
def test_portions_and_steps(kernels, shape, dtype, per_channel):
    H, G, D, DV, taps = shape
    T, slots = 150, 3
    on = _inputs(shape, per_channel, T, dtype, seed=sum(shape))
    cpu, gpu = on("cpu", torch.float32), on(DEV)
    C = 2 * G * D + H * DV
    state, ring = torch.full((slots, H, D, DV), 7.0, device=DEV), torch.full((slots, taps, C), 7.0, device=DEV).to(dtype)
    want_state, want_ring = torch.zeros(slots, H, D, DV), torch.zeros(slots, taps, C)
    seg = lambda at, n, dev: wa.ExtendBatch.build([[0]], [at], [n], 256, dev, state_slots=[1])  # noqa: E731
    want = delta.delta_extend(cpu, want_state, want_ring, seg(0, T, "cpu"))
    g = torch.Generator().manual_seed(1)
    z, w = torch.randn(T, H * DV + 8, generator=g).to(dtype), torch.randn(DV, generator=g).to(dtype)
    gated = delta.head_gate(want, z.float()[:, : H * DV], w.float(), "silu", 1e-3, 0.7)
    tol = 3e-5  # the recurrence is fp32 whatever the projections are
    for cuts in ([T], [2] * 75, [17, 1, 3, 64, 2, 1, 62], [100] + [1] * 50, [1] * 20 + [130]):
        at = 0
        state.fill_(7.0)
        ring.fill_(7.0)
        for n in cuts:
            if n == 1 and at > 0:
                i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
                rows = [0, at, 0]  # the outer rows are idle
                x = dataclasses.replace(gpu, **{f: torch.stack([getattr(gpu, f)[r] for r in rows]) for f in "qkvab"})
                x.q, x.k, x.v = torch.cat([x.q, x.k, x.v], 1).split([G * D, G * D, H * DV], 1)
                out = torch.full((3, H * DV + 16), 5.0, device=DEV).to(dtype)
                y = delta.delta_step(x, state, ring, i32(0, 1, 2), i32(0, 1, 0), i32(3, at, 3), z.to(DEV)[rows][:, : H * DV], w.to(DEV), "silu", 1e-3, 0.7,
                                     out[:, 8 : 8 + H * DV])
                _close(y[1], gated[at], 3e-5 if dtype == torch.float32 else 1e-2)
                assert float(y[[0, 2]].float().abs().max()) == 0 and float(out[:, :8].float().min()) == 5.0 == float(out[:, 8 + H * DV :].float().min())
            else:
                o = delta.delta_extend(_cut(gpu, at, at + n), state, ring, seg(at, n, DEV))
                _close(o, want[at : at + n], tol)
                _close(delta.head_gate(o, z.to(DEV)[at : at + n, : H * DV], w.to(DEV), "silu", 1e-3, 0.7), gated[at : at + n],
                       3e-5 if dtype == torch.float32 else 1e-2)
            at += n
        _close(state[1], want_state[1], tol)
        assert float((state[[0, 2]] - 7.0).abs().max()) == 0 and float((ring[[0, 2]].float() - 7.0).abs().max()) == 0  # others' slots
    o = torch.randn(5, H, DV, generator=g)
    _close(delta.head_gate(o.to(DEV), z.to(DEV)[:5, : H * DV], w.to(DEV), "sigmoid", 1e-3),
           delta.head_gate(o, z.float()[:5, : H * DV], w.float(), "sigmoid", 1e-3), 3e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("per_channel", [False, True])
def test_many_requests_in_one_pass(kernels, per_channel):
    """Portions of different lengths and ages side by side, slots in no order; the same rows alone give the same bits."""
    shape = H, G, D, DV, taps = (4, 2, 64, 80, 4)
    counts, starts, slots = [5, 1, 33, 16, 64, 2], [0, 9, 0, 40, 7, 1], [3, 0, 5, 1, 2, 4]
    on = _inputs(shape, per_channel, sum(counts), torch.bfloat16, seed=3)
    gpu, cpu = on(DEV), on("cpu", torch.float32)
    g = torch.Generator().manual_seed(4)
    s0, r0 = torch.randn(6, H, D, DV, generator=g), torch.randn(6, taps, 2 * G * D + H * DV, generator=g).bfloat16()
    build = lambda i, dev: wa.ExtendBatch.build([[0]] * len(i), [starts[j] for j in i], [counts[j] for j in i], 128, dev, state_slots=[slots[j] for j in i])  # noqa: E731,E501
    state, ring = s0.to(DEV), r0.to(DEV)
    got = delta.delta_extend(gpu, state, ring, build(range(6), DEV))
    ws, wr = s0.clone(), r0.float()
    want = delta.delta_extend(cpu, ws, wr, build(range(6), "cpu"))
    _close(got, want, 3e-5)
    _close(state, ws, 3e-5)
    assert torch.equal(ring.cpu().float(), wr)
    at = 0
    for i, n in enumerate(counts):
        s1, r1 = s0.to(DEV), r0.to(DEV)
        alone = delta.delta_extend(_cut(gpu, at, at + n), s1, r1, build([i], DEV))
        assert torch.equal(alone, got[at : at + n]) and torch.equal(s1[slots[i]], state[slots[i]]) and torch.equal(r1[slots[i]], ring[slots[i]])
        at += n


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", [(6, 2, 64, 64, 64, True), (4, 4, 48, 24, 20, True), (3, 1, 10, 14, 6, True), (8, 2, 128, 128, 32, False), (2, 2, 256, 16, 0, True)])
def test_heads_into_place(kernels, shape, dtype):
    Hq, Hkv, D, DV, dims, interleaved = shape
    g = torch.Generator().manual_seed(D)
    T, n = 29, Hq * D + Hkv * (D + DV)
    x = torch.randn(T, n + 8, generator=g).to(dtype)
    qn, kn = (torch.rand(D, generator=g).add(0.5).to(dtype) for _ in range(2))
    slots = torch.randperm(64, generator=g)[:T].to(torch.int32)
    slots[4] = -1
    pos = torch.randint(0, 500, (T,), generator=g, dtype=torch.int32)
    table = stream.rotary_table(500, dims, 1e4) if dims else None

    def run(dev, dt, norm):
        y = x.to(dev, dt, copy=True)
        kc, vc = torch.zeros(64, Hkv, D, dtype=dt, device=dev), torch.zeros(64, Hkv, DV, dtype=dt, device=dev)
        q, k, v, _ = y.split([Hq * D, Hkv * D, Hkv * DV, 8], 1)
        w = [t.to(dev, dt) for t in (qn, kn)] if norm else [None, None]
        out = stream.place_heads(q, k, v, slots.to(dev), kc, vc, q_norm=w[0], k_norm=w[1], eps=1e-2, table=None if table is None else table.to(dev),
                                 positions=pos.to(dev), interleaved=interleaved)
        return out, kc, vc

    for norm in (True, False):
        for got, want in zip(run(DEV, dtype, norm), run("cpu", torch.float32, norm)):
            _close(got, want, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtypes", [(torch.bfloat16, torch.bfloat16), (torch.float32, torch.float32), (torch.float32, torch.bfloat16)])
@pytest.mark.parametrize("H", [40, 45, 2048])
def test_pair_table_and_offset_norm(kernels, H, dtypes):
    ty, tw = dtypes
    g = torch.Generator().manual_seed(H)
    embed, table, w = torch.randn(300, H, generator=g).to(ty), torch.randn(102, H, generator=g).to(ty), (torch.randn(H, generator=g) * 0.3).to(tw)
    ids, prev = torch.randint(0, 300, (33,), generator=g, dtype=torch.int32), torch.randint(-1, 300, (33,), generator=g, dtype=torch.int32)
    for mp, mc in ((31, 7), (2**31 + 11, 2**33 + 1)):
        run = lambda d: stream.stream_norm(embed.to(d), None, w.to(d), 1e-3, ids=ids.to(d), offset=1.0, pair=stream.PairTable(table.to(d), ids.to(d), prev.to(d), mp, mc))  # noqa: E731,E501
        (h, res), (wh, wr) = run(DEV), run("cpu")
        assert torch.equal(res.cpu(), wr)
        _close(h, wh, 1e-5 if tw == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", [(6, 2, 64, 64, 64, None, 0), (5, 5, 40, 24, 16, None, 0), (8, 1, 128, 128, 64, 150, 3), (3, 1, 30, 50, 16, None, 0)])
def test_sinks_and_output_factor(kernels, shape, dtype):
    """With small scores the column without a value takes a visible share of every softmax; it must count once whatever the
    number of tiles and splits."""
    hq, hkv, d, dv, ps, window, keep = shape
    g = torch.Generator().manual_seed(d)
    starts, counts = [0, 700, 130, 0], [140, 1, 37, 2]
    need = [-(-(s + n) // ps) for s, n in zip(starts, counts)]
    order = torch.randperm(sum(need), generator=g).tolist()
    pages = [[order.pop() for _ in range(n)] for n in need]
    kc, vc = (torch.randn(sum(need) * ps, hkv, w, generator=g).to(dtype) for w in (d, dv))
    q = torch.randn(sum(counts), hq, d, generator=g).to(dtype)
    sinks = torch.linspace(-1.0, 7.0, hq)
    scale = 0.3 * d**-0.5
    run = lambda dev, dt: wa.window_extend(q.to(dev, dt), kc.to(dev, dt), vc.to(dev, dt), wa.ExtendBatch.build(pages, starts, counts, ps, dev), scale, window,  # noqa: E731,E501
                                           keep, sinks=sinks.to(dev), out_scale=-0.4)  # fmt: skip
    want = run("cpu", torch.float32)
    _close(run(DEV, dtype), want, 1e-5 if dtype == torch.float32 else 1e-2)
    plain = wa.window_extend(q.float(), kc.float(), vc.float(), wa.ExtendBatch.build(pages, starts, counts, ps, "cpu"), scale, window, keep, out_scale=-0.4)
    assert float((plain - want).abs().max()) > 0.05
    table = torch.zeros(4, max(need), dtype=torch.int32)
    for r, p in enumerate(pages):
        table[r, : len(p)] = torch.tensor(p)
    seq = torch.tensor([s + n for s, n in zip(starts, counts)], dtype=torch.int32)
    last = q[torch.tensor(counts).cumsum(0) - 1]
    rows = want[torch.tensor(counts).cumsum(0) - 1]
    for most in (None, 1 << 20):
        out = torch.zeros(4, hq * dv + 16, dtype=dtype, device=DEV)
        wa.window_decode(last.to(DEV), kc.to(DEV), vc.to(DEV), table.to(DEV), seq.to(DEV), (seq - 1).to(DEV), ps, scale, window, keep, sinks=sinks.to(DEV),
                         out_scale=-0.4, max_context=most, out=out[:, 8 : 8 + hq * dv])
        _close(out[:, 8 : 8 + hq * dv].reshape(4, hq, dv), rows, 1e-5 if dtype == torch.float32 else 1e-2)

"""Kernels of models with specified layers (fp32 residual stream, windowed attention, ungated experts) against plain fp32 torch."""

import pytest
import torch

from slime_b200 import ops
from slime_b200.ops import grouped, stream
from slime_b200.ops import window_attention as wa

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _norm(v, w, eps, kind):
    d = v - (v.mean(-1, keepdim=True) if kind == "layer" else 0)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


@pytest.mark.parametrize("H", [24, 100, 336, 1032, 2560, 8192])
@pytest.mark.parametrize("dtypes", [(torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16), (torch.float32, torch.float32)])
def test_stream_norm(kernels, H, dtypes):
    ty, tw = dtypes
    g = torch.Generator().manual_seed(H)
    T, eps = 37, 1e-4
    y = (torch.randn(T, H, generator=g) * 3 + 1.5).to(ty)
    res = torch.randn(T, H, generator=g)
    w1, w2 = (torch.randn(H, generator=g).to(tw) for _ in range(2))
    for kind in ("layer", "rms"):
        want_res = res + _norm(y.float(), w1.float(), eps, kind)
        want_h = _norm(want_res, w2.float(), eps, kind)
        r = res.to(DEV).clone()
        h, out = stream.stream_norm(y.to(DEV), r, w2.to(DEV), eps, kind=kind, post_w=w1.to(DEV))
        assert out is r and h.dtype == tw
        torch.testing.assert_close(r.cpu(), want_res, atol=2e-5, rtol=2e-5)
        tol = 2e-5 if tw == torch.float32 else 1e-2
        torch.testing.assert_close(h.float().cpu(), want_h, atol=tol, rtol=tol)
    table, ids = torch.randn(50, H, generator=g).to(ty), torch.randint(-3, 60, (T,), generator=g, dtype=torch.int32)
    rows = torch.where(((ids >= 0) & (ids < 50))[:, None], table.float()[ids.long().clamp(0, 49)], torch.zeros(T, H))
    h, r = stream.stream_norm(table.to(DEV), None, w2.to(DEV), eps, kind="layer", ids=ids.to(DEV))
    assert torch.equal(r.cpu(), rows)
    tol = 2e-5 if tw == torch.float32 else 1e-2
    torch.testing.assert_close(h.float().cpu(), _norm(rows, w2.float(), eps, "layer"), atol=tol, rtol=tol)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_expert_sum_in_the_norm(kernels, dtype):
    g = torch.Generator().manual_seed(1)
    T, k, H, R = 9, 3, 72, 40
    rows, shared = torch.randn(R, H, generator=g).to(dtype), torch.randn(T, H, generator=g).to(dtype)
    dest = torch.randint(-4, R, (T * k,), generator=g, dtype=torch.int32)
    wts, logits = torch.rand(T, k, generator=g), torch.randn(T, 8, generator=g)
    w = torch.rand(H, generator=g).to(dtype)
    cpu = stream.ExpertSum(rows, dest, wts, shared, logits[:, 5])
    gpu = stream.ExpertSum(rows.to(DEV), dest.to(DEV), wts.to(DEV), shared.to(DEV), logits.to(DEV)[:, 5])
    torch.testing.assert_close(stream.combine(gpu).cpu(), stream.combine(cpu), atol=1e-5, rtol=1e-5)
    res = torch.randn(T, H, generator=g)
    want = stream.stream_norm(cpu, res.clone(), w, 1e-5, kind="layer", post_w=w)
    got = stream.stream_norm(gpu, res.to(DEV), w.to(DEV), 1e-5, kind="layer", post_w=w.to(DEV))
    torch.testing.assert_close(got[1].cpu(), want[1], atol=2e-5, rtol=2e-5)
    torch.testing.assert_close(got[0].float().cpu(), want[0].float(), atol=2e-2, rtol=2e-2)


@pytest.mark.parametrize("act", ["silu", "gelu_tanh", "relu2"])
@pytest.mark.parametrize("F", [7, 48])
def test_activations(kernels, act, F):
    x = torch.randn(11, 2 * F, generator=torch.Generator().manual_seed(F)) * 3
    for gated in (True, False):
        for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
            want = stream.feed_forward_act(x.to(dt), act, gated).float()
            torch.testing.assert_close(stream.feed_forward_act(x.to(dt).to(DEV), act, gated).float().cpu(), want, atol=tol, rtol=tol)


@pytest.mark.parametrize("shape", [(1, 5, 3), (70, 130, 33), (129, 64, 320)])
def test_cuda_core_gemm(kernels, shape):
    M, N, K = shape
    g = torch.Generator().manual_seed(M)
    a, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    want = a.double() @ b.double().t()
    got = ops.gemm(a.to(DEV), b.to(DEV))
    assert float((got.cpu().double() - want).abs().max()) < 1e-5 * K**0.5
    ab, bb = a.bfloat16(), b.bfloat16()
    got = ops.gemm_simt(ab.to(DEV), bb.to(DEV), out_dtype=torch.float32)
    assert float((got.cpu().double() - ab.double() @ bb.double().t()).abs().max()) < 1e-5 * K**0.5


@pytest.mark.parametrize("E,k,T", [(5, 1, 3), (16, 3, 1), (40, 4, 77), (128, 8, 700), (6, 2, 0 + 33)])
def test_layout_kernel_matches_the_torch_layout(kernels, E, k, T):
    g = torch.Generator().manual_seed(E * T)
    idx = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).to(torch.int32)
    for n, first in ((E, 0), (max(E // 2, 1), E // 3)):
        a, b = grouped.DeviceLayout(idx, n, first), grouped.DeviceLayout(idx.to(DEV), n, first)
        assert a.rows_padded == b.rows_padded
        assert torch.equal(a.slot_dest, b.slot_dest.cpu()) and torch.equal(a.tile_expert, b.tile_expert.cpu())


@pytest.mark.parametrize("dtype,dims", [(torch.float32, (33, 20, 57)), (torch.bfloat16, (64, 40, 56)), (torch.bfloat16, (36, 20, 36))])
def test_ungated_experts(kernels, dtype, dims):
    """Routing, permutation, both grouped products and the weighted sum; the last shape has rows no TMA descriptor takes."""
    H, F, _ = dims
    E, k, T = 6, 2, 50
    g = torch.Generator().manual_seed(3)
    x, w1, w2 = torch.randn(T, H, generator=g), torch.randn(E, F, H, generator=g) * 0.2, torch.randn(E, H, F, generator=g) * 0.2
    logits = torch.randn(T, 8, generator=g)
    x, w1, w2 = x.to(dtype), w1.to(dtype), w2.to(dtype)
    score = logits[:, :E].softmax(-1)
    top = score.topk(k, -1)
    want = torch.zeros(T, H)
    for t in range(T):
        for j in range(k):
            e = int(top.indices[t, j])
            want[t] += top.values[t, j] * ((x[t].float() @ w1[e].float().t()).clamp_min(0).square() @ w2[e].float().t())
    probs, idx = grouped.route_topk(logits.to(DEV)[:, :E], k, renorm=False, raw_index=True)
    lay = grouped.DeviceLayout(idx, E)
    up = grouped.grouped_gemm(lay.pad(x.to(DEV)), w1.to(DEV), lay)
    rows = grouped.grouped_gemm(stream.feed_forward_act(up, "relu2", False), w2.to(DEV), lay)
    got = stream.combine(stream.ExpertSum(rows, lay.slot_dest, probs)).cpu()
    scale = float(want.abs().max())
    assert float((got - want).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2) * scale


def _cache(g, reqs, hkv, d, dv, ps, dtype, spare=3):
    """Keys / values of ``reqs`` (lengths) in shuffled pages of a pool whose other pages hold large finite garbage."""
    need = [-(-n // ps) for n in reqs]
    order = (torch.randperm(sum(need) + spare, generator=g)).tolist()
    table, at = torch.zeros(len(reqs), max(need), dtype=torch.int32), 0
    kc = torch.full(((sum(need) + spare) * ps, hkv, d), 1e4).to(dtype)
    vc = torch.full(((sum(need) + spare) * ps, hkv, dv), -1e4).to(dtype)
    for r, n in enumerate(reqs):
        pages = order[at : at + need[r]]
        at += need[r]
        table[r, : need[r]] = torch.tensor(pages, dtype=torch.int32)
        slots = torch.tensor([pages[p // ps] * ps + p % ps for p in range(n)])
        kc[slots], vc[slots] = torch.randn(n, hkv, d, generator=g).to(dtype), torch.randn(n, hkv, dv, generator=g).to(dtype)
    return kc, vc, table


SHAPES = [  # heads, kv heads, dim, vdim, page, window, keep
    (8, 2, 64, 64, 16, 40, 3), (4, 4, 128, 128, 64, 200, 0), (6, 2, 48, 72, 32, 129, 5), (7, 1, 64, 128, 16, 128, 130), (16, 1, 80, 16, 128, 1, 0),
    (12, 4, 128, 64, 64, None, 0), (40, 1, 64, 64, 16, 77, 9), (5, 5, 40, 40, 64, 300, 1), (3, 1, 30, 50, 16, 33, 2), (2, 1, 160, 256, 32, 65, 4),
]  # fmt: skip


def _check(got, want, dtype):
    err = float((got.float().cpu() - want.float()).abs().max())
    assert err < (2e-5 if dtype == torch.float32 else 2e-2) * max(1.0, float(want.float().abs().max())), err


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bias", [True, False])
def test_window_attention_of_portions_and_single_tokens(kernels, shape, dtype, bias):
    hq, hkv, d, dv, ps, window, keep = shape
    g = torch.Generator().manual_seed(sum(shape[:5]))
    starts, counts = [0, 517, 130, 0, 63, 299], [150, 1, 37, 1, 2, 133]
    kc, vc, table = _cache(g, [s + n for s, n in zip(starts, counts)], hkv, d, dv, ps, dtype)
    pages = [table[r, : -(-(s + n) // ps)].tolist() for r, (s, n) in enumerate(zip(starts, counts))]
    T = sum(counts)
    qkv = torch.randn(T, hq * d + 16, generator=g).to(dtype)
    q = qkv[:, : hq * d].unflatten(1, (hq, d))
    slopes = torch.tensor([2.0 ** (-8 * (h + 1) / hq) for h in range(hq)]) if bias else None
    args = (0.7 * d**-0.5, window, keep)
    want = wa.window_extend(q.float(), kc.float(), vc.float(), wa.ExtendBatch.build(pages, starts, counts, ps, "cpu"), *args, slopes)
    qd = qkv.to(DEV)[:, : hq * d].unflatten(1, (hq, d))
    got = wa.window_extend(qd, kc.to(DEV), vc.to(DEV), wa.ExtendBatch.build(pages, starts, counts, ps, DEV), *args,
                           None if slopes is None else slopes.to(DEV))
    _check(got, want, dtype)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_of_decode_steps(kernels, shape, dtype):
    hq, hkv, d, dv, ps, window, keep = shape
    g = torch.Generator().manual_seed(sum(shape[:5]))
    lens = [1, 2, 63, 64, 65, 128, 129, 200, 201, 257, 700, 1111]
    kc, vc, table = _cache(g, lens, hkv, d, dv, ps, dtype)
    q = torch.randn(len(lens), hq, d, generator=g).to(dtype)
    slopes = torch.tensor([2.0 ** (-8 * (h + 1) / hq) for h in range(hq)])
    seq = torch.tensor(lens, dtype=torch.int32)
    args = (ps, 0.7 * d**-0.5, window, keep)
    want = wa.window_decode(q.float(), kc.float(), vc.float(), table, seq, seq - 1, *args, slopes)
    dev = [x.to(DEV) for x in (q, kc, vc, table, seq, seq - 1)]
    for most in (None, 1 << 20):  # different split counts
        _check(wa.window_decode(*dev, *args, slopes.to(DEV), max_context=most), want, dtype)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_one_key_stands_out_at_every_edge(kernels, dtype):
    """One key matches the query strongly; it must count exactly when it is inside the window or kept, whatever the tile,
    page and portion it falls into. Values name their position, so the answer is the position of the key that won."""
    ps, window, keep, n, d = 16, 70, 5, 333, 64
    pages = [torch.randperm(40, generator=torch.Generator().manual_seed(0))[: -(-n // ps)].tolist()]
    slots = torch.tensor([pages[0][p // ps] * ps + p % ps for p in range(n)])
    for pos in (69, 70, 75, 127, 128, 200, 255, 256, 332):
        for key in {0, 4, 5, pos - 71, pos - 70, pos - 69, pos - 1, pos} - {k for k in range(-100, 0)}:
            kc, vc = torch.zeros(40 * ps, 1, d), torch.zeros(40 * ps, 1, 64)
            kc[slots[key], 0, 0] = 30.0
            vc[slots[key], 0, 0] = 1.0
            q = torch.zeros(2, 1, d)
            q[:, 0, 0] = 1.0
            seen = key <= pos and (pos - key < window or key < keep)
            dev = [x.to(DEV, dtype) for x in (q[:1], kc, vc)]
            b = wa.ExtendBatch.build(pages, [pos], [1], ps, DEV)
            one = wa.window_extend(*dev, b, 1.0, window, keep)[0, 0, 0]
            s = torch.tensor([pos + 1], dtype=torch.int32, device=DEV)
            dec = wa.window_decode(*dev, b.block_table, s, s - 1, ps, 1.0, window, keep)[0, 0, 0]
            for v in (one, dec):
                assert abs(float(v) - float(seen)) < 1e-2, (pos, key, seen, float(v))

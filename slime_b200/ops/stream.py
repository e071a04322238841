"""Ops around an fp32 residual stream (``csrc/stream.cu``): the fused step between two sub-layers of a decoder that
normalises before each of them, behind it, or both, feed-forward activations, and cache writes of any width.

CUDA tensors run the kernels; CPU tensors run the definitions in this file.
"""

from __future__ import annotations

import dataclasses

import torch

from slime_b200.ops import _checks, _lib

P = _lib.ptr
ACTS = {"silu": 0, "gelu_tanh": 1, "relu2": 2}


@dataclasses.dataclass
class ExpertSum:
    """Unfinished output of a mixture-of-experts feed-forward: token t is ``sum_j weights[t, j] * rows[dest[t * k + j]]``
    (``dest`` < 0: no row here) ``+ sigmoid(gate[t]) * shared[t] + base[t]``. ``gate``: a column of the router's logits, or None;
    ``base``: fp32 output of what runs beside the experts, or None."""

    rows: torch.Tensor
    dest: torch.Tensor
    weights: torch.Tensor
    shared: torch.Tensor | None = None
    gate: torch.Tensor | None = None
    base: torch.Tensor | None = None

    def tokens(self) -> int:
        return self.weights.shape[0]


@dataclasses.dataclass
class PairTable:
    """Second embedding table: token t adds row ``(prev * mul_prev + token * mul_cur) mod (rows - 1)`` of ``table``, the last row
    where it has no predecessor (``prev`` < 0)."""

    table: torch.Tensor
    ids: torch.Tensor
    prev: torch.Tensor
    mul_prev: int
    mul_cur: int

    def rows(self) -> torch.Tensor:
        n = self.table.shape[0] - 1
        r = (self.prev.long() * self.mul_prev + self.ids.long() * self.mul_cur) % n
        return torch.where(self.prev >= 0, r, torch.full_like(r, n))


def _norm(v, w, eps, kind, offset=0.0, groups=1):
    if groups > 1:
        p = v.unflatten(-1, (groups, -1))
        return (p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * (w.float() + offset)
    mean = v.mean(-1, keepdim=True) if kind == "layer" else 0.0
    d = v - mean
    return d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps) * (w.float() + offset)


def _combine(e: ExpertSum) -> torch.Tensor:
    T, k = e.weights.shape
    d = e.dest.view(T, k).long()
    y = torch.zeros(T, e.rows.shape[-1], dtype=torch.float32, device=e.rows.device)
    for j in range(k):
        hit = (d[:, j] >= 0)[:, None]
        y += torch.where(hit, e.weights[:, j : j + 1].float() * e.rows[d[:, j].clamp_min(0)].float(), torch.zeros_like(y))
    if e.shared is not None:
        s = e.shared.float()
        y += s if e.gate is None else torch.sigmoid(e.gate.float())[:, None] * s
    return y if e.base is None else y + e.base


def stream_norm(y, res, pre_w, eps, *, kind="rms", post_w=None, ids=None, offset=0.0, pair: PairTable | None = None,
                gain=1.0, groups=1, emit: torch.dtype | None = None):  # fmt: skip
    """``res (+)= norm(y) * post_w`` and return ``norm(res) * pre_w``, in one launch.

    ``y``: sub-layer output [T, H], an ``ExpertSum``, or an embedding table when ``ids`` [T] is given (ids outside the table give
    zero rows: other ranks' part of a sharded vocabulary). ``res``: fp32 [T, H],
    updated in place; None starts the stream (a new tensor is returned as second value). ``post_w`` None: no norm of the
    sub-layer's output; ``pre_w`` None: nothing but the stream is wanted (the first value is None), or with ``emit`` the stream itself in
    that type. ``kind``: "rms" or "layer" (mean removed, no bias); ``groups``: equal parts of a row with an RMS norm of their own; ``offset`` is added to the norm weights in fp32. ``pair``: rows of a second table added to
    ``y``. ``gain``: factor of the first value. Norms, sums and the stream are fp32 whatever the element types."""
    moe = y if isinstance(y, ExpertSum) else None
    src = moe.rows if moe is not None else y
    T = moe.tokens() if moe is not None else (ids.numel() if ids is not None else y.shape[0])
    H = src.shape[-1]
    init = res is None
    if moe is not None:
        _checks.index_range("stream_norm", "dest", moe.dest, upper=src.shape[0], lower=-(1 << 31))
    w_dtype = pre_w.dtype if pre_w is not None else emit or (post_w.dtype if post_w is not None else src.dtype)
    assert kind == "rms" or groups == 1
    if not src.is_cuda:
        if ids is not None:
            i = ids.long()
            v = src[i.clamp(0, src.shape[0] - 1)].float() * ((i >= 0) & (i < src.shape[0]))[:, None]
        else:
            v = _combine(moe) if moe is not None else src.float()
        if pair is not None:
            v = v + pair.table[pair.rows()].float()
        if post_w is not None:
            v = _norm(v, post_w, eps, kind, offset, groups)
        if init:
            res = v.clone()
        else:
            res.add_(v)
        if pre_w is None and emit is None:
            return None, res
        h = res if pre_w is None else _norm(res, pre_w, eps, kind, offset, groups)
        return (h * gain).to(w_dtype), res
    src = src.contiguous()
    if init:
        res = torch.empty(T, H, dtype=torch.float32, device=src.device)
    assert res.dtype == torch.float32 and res.is_contiguous() and src.dtype in (torch.bfloat16, torch.float32)
    h = torch.empty(T, H, dtype=w_dtype, device=src.device) if pre_w is not None or emit is not None else None
    assert all(w is None or w.dtype == w_dtype for w in (pre_w, post_w))
    dest = wts = shared = gate = base = None
    k = 1
    if moe is not None:
        k = moe.weights.shape[1]
        dest, wts = moe.dest.contiguous(), moe.weights.contiguous()
        assert dest.dtype == torch.int32 and wts.dtype == torch.float32
        shared = None if moe.shared is None else moe.shared.contiguous()
        assert shared is None or shared.dtype == src.dtype
        gate = moe.gate if shared is not None else None
        assert gate is None or gate.dtype == torch.float32
        base = moe.base
        assert base is None or (base.dtype == torch.float32 and base.is_contiguous() and base.shape == (T, H))
    ids32 = None if ids is None else ids.to(torch.int32).contiguous()
    if pair is not None:
        assert pair.table.is_contiguous() and pair.table.dtype == src.dtype and pair.table.shape[1] == H
        assert pair.ids.dtype == pair.prev.dtype == torch.int32 and pair.ids.is_contiguous() and pair.prev.is_contiguous()
    rc = _lib.lib().sb_stream_norm(
        P(src), int(src.dtype == torch.float32), P(ids32), src.shape[0], P(dest), P(wts), k, P(shared), P(gate),
        gate.stride(0) if gate is not None else 0, P(post_w), P(res), int(init), P(pre_w), P(h), int(w_dtype == torch.float32),
        T, H, float(eps), float(offset), int(kind == "layer"), P(pair.table) if pair else None, P(pair.ids) if pair else None,
        P(pair.prev) if pair else None, pair.mul_prev if pair else 0, pair.mul_cur if pair else 0, pair.table.shape[0] - 1 if pair else 0,
        P(base), float(gain), int(groups), _lib.stream(),
    )  # fmt: skip
    _lib.check(rc, "sb_stream_norm")
    return h, res


def combine(e: ExpertSum) -> torch.Tensor:
    """The sum an ``ExpertSum`` stands for, fp32 [T, H] (where a collective has to come before the norm)."""
    return stream_norm(e, None, None, 0.0)[1]


def feed_forward_act(x: torch.Tensor, act: str, gated: bool, out: torch.Tensor | None = None) -> torch.Tensor:
    """``act(x[:, :F]) * x[:, F:]`` (gated) or ``act(x)``; ``x`` and ``out`` may be column ranges of wider matrices."""
    F = x.shape[-1] // 2 if gated else x.shape[-1]
    if not x.is_cuda:
        g = x[..., :F].float()
        if act == "silu":
            g = g * torch.sigmoid(g)
        elif act == "gelu_tanh":
            g = torch.nn.functional.gelu(g, approximate="tanh")
        else:
            g = g.clamp_min(0).square()
        y = (g * x[..., F:].float() if gated else g).to(x.dtype)
        return y if out is None else out.copy_(y)
    x = x if x.stride(-1) == 1 else x.contiguous()
    if out is None:
        out = torch.empty(x.shape[0], F, dtype=x.dtype, device=x.device)
    assert out.dtype == x.dtype and out.stride(-1) == 1 and out.shape == (x.shape[0], F)
    rc = _lib.lib().sb_glu(P(x), P(x[:, F:]) if gated else None, P(out), x.shape[0], F, x.stride(0), out.stride(0), ACTS[act],
                           int(x.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_glu")
    return out


def poly_sums(x: torch.Tensor) -> torch.Tensor:
    """[T, 3] fp32 sums of the second, fourth and sixth powers of rows (a rank's part of them)."""
    p = x.float().square()
    return torch.stack([p.sum(-1), p.square().sum(-1), (p.square() * p).sum(-1)], 1)


def poly_norm(x: torch.Tensor, coef: torch.Tensor, eps: float, sums: torch.Tensor | None = None, width: int | None = None) -> torch.Tensor:
    """``a N(x) + b N(x^2) + c N(x^3) + e`` of whole rows with (a, b, c, e) = ``coef`` (fp32) and N dividing a row by its root mean square. ``sums``,
    ``width``: power sums and width of the whole rows, of which ``x`` is a part."""
    T, F = x.shape
    width = width or F
    if not x.is_cuda:
        z, s = x.float(), poly_sums(x) if sums is None else sums
        r = coef[:3] * torch.rsqrt(s / width + eps)
        return (((z * r[:, 2:3] + r[:, 1:2]) * z + r[:, 0:1]) * z + coef[3]).to(x.dtype)
    x = x if x.stride(1) == 1 else x.contiguous()
    assert coef.dtype == torch.float32 and coef.numel() == 4 and (sums is None or (sums.is_contiguous() and sums.shape == (T, 3)))
    out = torch.empty(T, F, dtype=x.dtype, device=x.device)
    rc = _lib.lib().sb_poly_norm(P(x), P(out), P(coef), P(sums), T, F, width, x.stride(0), out.stride(0), float(eps), int(x.dtype == torch.float32),
                                 _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_poly_norm")
    return out


def softcap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap tanh(x / cap)`` in place (fp32 rows)."""
    if not x.is_cuda:
        return x.div_(cap).tanh_().mul_(cap)
    assert x.dtype == torch.float32 and x.stride(1) == 1
    for part in x.split(65535):
        _lib.check(_lib.lib().sb_softcap(P(part), part.shape[0], part.shape[1], part.stride(0), float(cap), _lib.stream()), "sb_softcap")
    return x


def rotary_table(positions: int, dims: int, base: float, device=None, *, frequencies: list[float] | None = None, gain: float = 1.0) -> torch.Tensor:
    """fp32 ``[positions, dims]`` = cos | sin of ``p * base^(-2i / dims)`` for the dims / 2 pairs i (computed in fp64); ``frequencies``:
    those instead; ``gain`` multiplies the table."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if frequencies is not None:
        f = torch.tensor(frequencies, dtype=torch.float64)
    angle = torch.arange(positions, dtype=torch.float64)[:, None] * f
    return (torch.cat([angle.cos(), angle.sin()], 1) * gain).float().to(device)


def _turn(x, table, positions, interleaved):
    half = table.shape[1] // 2
    cos, sin = table[positions.long()][:, None].split(half, dim=-1)
    pair = slice(0, 2 * half, 2), slice(1, 2 * half, 2)
    if not interleaved:
        pair = slice(0, half), slice(half, 2 * half)
    out = x.clone()
    u, v = x[..., pair[0]], x[..., pair[1]]
    out[..., pair[0]], out[..., pair[1]] = u * cos - v * sin, v * cos + u * sin
    return out


def place_heads(q, k, v, slots, k_cache, v_cache, *, q_norm=None, k_norm=None, eps=0.0, table=None, positions=None, interleaved=True,
                sums=None, maps=1):  # fmt: skip
    """New queries ``q`` [T, Hq * D], keys [T, Hkv * D] and values [T, Hkv * DV] (column ranges of a projection are fine; values may be
    the keys): RMS norm (``q_norm`` / ``k_norm`` [D]: per query / key head; [Hq * D] / [Hkv * D]: over all heads at once; None: none),
    rotation by ``table`` (``rotary_table``; None: none) at ``positions``. Queries are changed in place and returned [T, Hq, D]; keys
    and values go to cache slot ``slots[t]`` (< 0: nowhere). ``sums``: for a norm over all heads of which this rank has a part,
    ([T, 2] sums of squares of the whole projections, their widths). ``k``, ``v`` None: the cache has them already.

    ``maps`` 2 (differential attention): every head of the cache holds two keys of width D side by side, queries come in pairs of heads of
    width D that meet one of them each. They are returned [T, Hq, 2 D] with zeros where the other key stands."""
    if maps == 2:
        return _place_pairs(q, k, v, slots, k_cache, v_cache, q_norm, k_norm, eps, table, positions, interleaved)
    T, (Hkv, D), DV = q.shape[0], k_cache.shape[1:], v_cache.shape[2]
    Hq = q.shape[1] // D
    over_all = q_norm is not None and k_norm is not None and q_norm.numel() == Hq * D and k_norm.numel() == Hkv * D and (Hq > 1 or Hkv > 1 or sums is not None)
    _checks.index_range("place_heads", "slots", slots, upper=k_cache.shape[0], lower=-(1 << 31))
    if table is not None:
        _checks.index_range("place_heads", "positions", positions, upper=table.shape[0])
    if q_norm is None and table is None:
        if k is not None:
            kv_scatter(k, v, slots, k_cache, v_cache)
        return q.unflatten(1, (Hq, D))
    assert k is not None or not over_all
    if not q.is_cuda:
        out = []
        for i, (x, w) in enumerate(((q, q_norm), (k, k_norm)) if k is not None else ((q, q_norm),)):
            if over_all and sums is not None:
                x = (x.float() * torch.rsqrt(sums[0][:, i : i + 1] / sums[1][i] + eps) * w.float()).unflatten(1, (-1, D))
            elif over_all:
                x = _norm(x.float(), w, eps, "rms").unflatten(1, (-1, D))
            else:
                x = x.unflatten(1, (-1, D)).float()
                x = x if w is None else _norm(x, w, eps, "rms")
            out.append((x if table is None else _turn(x, table, positions, interleaved)).flatten(1).to(q.dtype))
        q.copy_(out[0])
        if k is not None:
            kv_scatter(out[1], v, slots, k_cache, v_cache)
        return q.unflatten(1, (Hq, D))
    f32 = int(q.dtype == torch.float32)
    if not over_all:
        _heads(q, k, v, q, slots, k_cache, v_cache, q_norm, k_norm, eps, table, positions, interleaved, (Hq, Hkv, Hkv, D, DV), 1)
        return q.unflatten(1, (Hq, D))
    _check_heads(q, k, v, k_cache, v_cache, q_norm, k_norm)
    head = (P(q), P(k), P(v), P(q_norm), P(k_norm), P(table), P(positions), P(slots), P(k_cache), P(v_cache), T, Hq, Hkv, D, DV,
            0 if table is None else table.shape[1], int(interleaved), q.stride(0), k.stride(0), v.stride(0))  # fmt: skip
    part, widths = sums if sums is not None else (None, (Hq * D, Hkv * D))
    _lib.check(_lib.lib().sb_heads_all(*head, P(part), *widths, float(eps), f32, _lib.stream()), "sb_heads_all")
    return q.unflatten(1, (Hq, D))


def _check_heads(q, k, v, k_cache, v_cache, q_norm, k_norm):
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and q.stride(1) == 1 and q.dtype == k_cache.dtype == v_cache.dtype
    assert all(x is None or (x.stride(-1) == 1 and x.dtype == q.dtype) for x in (k, v, q_norm, k_norm))


def _heads(q, k, v, q_out, slots, k_cache, v_cache, q_norm, k_norm, eps, table, positions, interleaved, sizes, maps):
    _check_heads(q, k, v, k_cache, v_cache, q_norm, k_norm)
    Hq, Hkv, Hv, D, DV = sizes
    if k is None:
        Hkv = Hv = 0
    rc = _lib.lib().sb_heads(
        P(q), P(k), P(v), P(q_out), P(q_norm), P(k_norm), P(table), P(positions), P(slots), P(k_cache), P(v_cache), q.shape[0], Hq, Hkv, Hv, D, DV,
        0 if table is None else table.shape[1], int(interleaved), maps, q.stride(0), 0 if k is None else k.stride(0), 0 if v is None else v.stride(0),
        q_out.stride(0), float(eps), int(q.dtype == torch.float32), _lib.stream(),
    )  # fmt: skip
    _lib.check(rc, "sb_heads")


def _place_pairs(q, k, v, slots, k_cache, v_cache, q_norm, k_norm, eps, table, positions, interleaved):
    T, (G, D2), (Hv, DV) = q.shape[0], k_cache.shape[1:], v_cache.shape[1:]
    D = D2 // 2
    Hq = q.shape[1] // D
    assert D2 == 2 * D and G == Hv and Hq % 2 == 0
    _checks.index_range("place_heads", "slots", slots, upper=k_cache.shape[0], lower=-(1 << 31))
    if table is not None:
        _checks.index_range("place_heads", "positions", positions, upper=table.shape[0])
    if not q.is_cuda:
        out = []
        for x, w in ((q, q_norm), (k, k_norm)) if k is not None else ((q, q_norm),):
            x = x.unflatten(1, (-1, D)).float()
            x = x if w is None else _norm(x, w, eps, "rms")
            out.append((x if table is None else _turn(x, table, positions, interleaved)).to(q.dtype))
        if k is not None:
            kv_scatter(out[1].flatten(1), v, slots, k_cache, v_cache)
        wide = torch.zeros(T, Hq, 2, D, dtype=q.dtype)
        wide[:, 0::2, 0], wide[:, 1::2, 1] = out[0][:, 0::2], out[0][:, 1::2]
        return wide.flatten(2)
    wide = torch.empty(T, Hq * D2, dtype=q.dtype, device=q.device)
    _heads(q, k, v, wide, slots, k_cache, v_cache, q_norm, k_norm, eps, table, positions, interleaved, (Hq, 2 * G, Hv, D, DV), 2)
    return wide.unflatten(1, (Hq, D2))


def head_sums(q, k) -> torch.Tensor:
    """[T, 2] fp32 sums of squares of query and key rows (a rank's part of them)."""
    return torch.stack([q.float().square().sum(-1), k.float().square().sum(-1)], 1)


def kv_scatter(k, v, slots, k_cache, v_cache):
    """Rows ``k[t]`` [Hkv * D] and ``v[t]`` [Hkv * DV] (views with any row pitch) into cache slot ``slots[t]`` (< 0: skipped)."""
    _checks.index_range("kv_scatter", "slots", slots, upper=k_cache.shape[0], lower=-(1 << 31))
    if not k.is_cuda:
        ok = slots >= 0
        for src, dst in ((k, k_cache), (v, v_cache)):
            dst.view(dst.shape[0], -1)[slots[ok].long()] = src[ok].to(dst.dtype)
        return
    assert k.stride(1) == 1 and v.stride(1) == 1 and k.dtype == k_cache.dtype and v.dtype == v_cache.dtype
    assert k_cache.is_contiguous() and v_cache.is_contiguous()
    es = k.element_size()
    rc = _lib.lib().sb_kv_scatter(P(k), P(v), P(slots), P(k_cache), P(v_cache), k.shape[0], k.shape[1] * es, v.shape[1] * es,
                                  k.stride(0) * es, v.stride(0) * es, _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_kv_scatter")

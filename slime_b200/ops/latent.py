"""Latent attention over the paged cache: one vector per token, the normed key/value latent [R2] and a rotated key part [r] that all
heads share (cache [slots, 1, R2 + r]).

Per head the unrotated key is ``up_k c`` and the value ``up_v c``. A query sees its context in one of two forms:

* absorbed: the query takes the key expansion on itself, ``q_lat = up_k^T q``, so scores and the weighted sum are formed with the
  cached vectors as they are, and ``up_v`` is applied to the result. Decode steps and short portions.
* expanded: the context's keys and values are expanded once per pass and head, then attention is the ordinary one with heads of
  D + r / DV. Long portions: per (query, key) pair it costs D + r + DV instead of 2 R2 + r multiplications.

CUDA tensors run the kernels (``csrc/latent_sm100.cu``, ``csrc/flash_window_sm100.cu``, ``csrc/stream.cu``; fp32 and shapes the tensor-core
kernels do not take: ``csrc/window_attn.cu``, ``csrc/gemm_simt.cu``); CPU tensors run the definitions in this file.
"""

from __future__ import annotations

import ctypes
import dataclasses

import torch

from slime_b200.ops import _checks, _lib, stream
from slime_b200.ops import window_attention as wa

P = _lib.ptr
EXPAND_FROM = 64  # new tokens of a request from which expanding its context is the cheaper form


def latent_place(dq, dkv, q_norm, kv_norm, eps, table, positions, slots, cache, interleaved=False):
    """New tokens' down-projections ``dq`` [T, R1] and ``dkv`` [T, R2 + r] (column ranges are fine) -> normed query latents [T, R1]; the
    normed key/value latent and the rotated shared key go to cache row ``slots[t]`` (< 0: nowhere)."""
    T, R1, R2, r = dq.shape[0], q_norm.numel(), kv_norm.numel(), table.shape[1]
    assert cache.shape[1:] == (1, R2 + r) and cache.is_contiguous()
    _checks.index_range("latent_place", "slots", slots, upper=cache.shape[0], lower=-(1 << 31))
    _checks.index_range("latent_place", "positions", positions, upper=table.shape[0])
    if not dq.is_cuda:
        c = stream._norm(dkv[:, :R2].float(), kv_norm, eps, "rms")
        k = stream._turn(dkv[:, None, R2:].float(), table, positions, interleaved)[:, 0]
        ok = slots >= 0
        cache[slots[ok].long(), 0] = torch.cat([c, k], 1)[ok].to(cache.dtype)
        return stream._norm(dq.float(), q_norm, eps, "rms").to(dq.dtype)
    assert dq.stride(1) == dkv.stride(1) == 1 and dq.dtype == dkv.dtype == cache.dtype == q_norm.dtype == kv_norm.dtype
    out = torch.empty(T, R1, dtype=dq.dtype, device=dq.device)
    rc = _lib.lib().sb_latent_place(P(dq), P(dkv), P(q_norm), P(kv_norm), P(table), P(positions), P(slots), P(out), P(cache), T, R1, R2, r,
                                    int(interleaved), dq.stride(0), dkv.stride(0), float(eps), int(dq.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_latent_place")
    return out


def turn_into(q, dst, table, positions, interleaved=False):
    """The last r coordinates of every head of ``q`` [T, H, D + r], rotated, into ``dst`` [T, H, r] (a view; it may be those coordinates)."""
    T, H, W = q.shape
    r = table.shape[1]
    if not q.is_cuda:
        dst.copy_(stream._turn(q[..., W - r :].float(), table, positions, interleaved).to(dst.dtype))
        return
    assert q.stride(2) == dst.stride(2) == 1 and q.dtype == dst.dtype
    rc = _lib.lib().sb_latent_turn(P(q), P(dst), P(table), P(positions), T, H, W - r, r, int(interleaved), q.stride(0), q.stride(1), dst.stride(0),
                                   dst.stride(1), int(q.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_latent_turn")


def head_gemm(x, w, out, *, transposed=False, gate=None):
    """``out[:, h] = x[:, h] @ w[h]^T`` (``w`` [H, N, K]) or ``@ w[h]`` (``transposed``, ``w`` [H, K, N]), times ``sigmoid(gate[:, h])``.
    ``x`` [T, H, K], ``out`` [T, H, N] and ``gate`` [T, H, N] may be views with any row and head pitch."""
    T, H, K = x.shape
    N = out.shape[2]
    assert w.shape == ((H, K, N) if transposed else (H, N, K)) and out.shape == (T, H, N) and w.stride(2) == 1
    if not x.is_cuda:
        y = torch.einsum("thk,hkn->thn" if transposed else "thk,hnk->thn", x.float(), w.float())
        out.copy_((y if gate is None else y * torch.sigmoid(gate.float())).to(out.dtype))
        return out
    assert x.stride(2) == out.stride(2) == 1 and x.dtype == w.dtype == out.dtype and (gate is None or (gate.stride(2) == 1 and gate.dtype == x.dtype))
    g = (0, 0) if gate is None else (gate.stride(0), gate.stride(1))
    args = (P(x), P(w), P(out), P(gate), H, T, N, K, int(transposed), x.stride(0), x.stride(1), w.stride(0), w.stride(1), out.stride(0), out.stride(1), *g)
    if x.dtype == torch.bfloat16:
        rc = _lib.lib().sb_head_gemm(*args, P(_lib.status_word(x.device)), _lib.stream())
        if rc != -1:  # -1: a width or an alignment the tensor-core kernel does not take
            _lib.check(rc, "sb_head_gemm")
            return out
    _lib.check(_lib.lib().sb_gemm_simt_heads(*args, int(x.dtype == torch.float32), _lib.stream()), "sb_gemm_simt_heads")
    return out


def latent_rows(q, cache, R2, block_table, row_req, positions, page_size, scale, max_context, out=None):
    """Absorbed attention: row t of ``q`` [T, H, R2 + r] stands at ``positions[t]`` of request ``row_req[t]`` (None: request t) and sees all
    earlier vectors of the cache -> [T, H, R2]."""
    T, H, W = q.shape
    if not q.is_cuda:
        return wa._reference(q, cache, cache[..., :R2], block_table, row_req, positions, page_size, scale)
    assert q.is_contiguous() and cache.is_contiguous()
    out = torch.empty(T, H, R2, dtype=q.dtype, device=q.device) if out is None else out
    if q.dtype == torch.bfloat16:
        longest = min(max_context, block_table.shape[1] * page_size)
        heads = 16 if H <= 16 else 32
        splits = wa.decode_splits(T, -(-H // heads), longest, q.device, resident=1, tile=64, limit=32)
        n = T * H * splits  # partial (maximum, sum) pairs come first: they are read as pairs
        ml = torch.empty(n * (R2 + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
        part = ml[2 * n :] if splits > 1 else None
        rule = wa.Rule.of(q, R2, scale)
        rc = _lib.lib().sb_latent_attn(P(q), P(cache), P(block_table), P(row_req), P(positions), P(out), P(part), P(ml), T, H, R2, W, page_size,
                                       block_table.stride(0), cache.shape[0], heads, splits, ctypes.byref(rule), P(_lib.status_word(q.device)),
                                       _lib.stream())  # fmt: skip
        if rc != -1:
            _lib.check(rc, "sb_latent_attn")
            return out
    return wa.simt(q, cache, cache[..., :R2], block_table, row_req, positions, page_size, wa.Rule.of(q, R2, scale), out)


@dataclasses.dataclass
class Latent:
    """Sizes and matrices of a latent mixer: ``up_q`` [H * (D + r), R1], ``up_kv`` [H * D + H * DV, R2] (keys first), ``table``: its
    rotation."""

    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float
    up_q: torch.Tensor
    up_kv: torch.Tensor
    table: torch.Tensor
    interleaved: bool = False

    @property
    def up_k(self):
        return self.up_kv[: self.heads * self.dim].view(self.heads, self.dim, self.rank)

    @property
    def up_v(self):
        return self.up_kv[self.heads * self.dim :].view(self.heads, self.vdim, self.rank)

    def absorbed(self, q, positions, attend, gate, out):
        """``q`` [T, H, D + r] (not yet rotated) through ``attend(q_lat) -> [T, H, R2]``; result times sigmoid(gate) into ``out`` [T, H, DV]."""
        T, H, W = q.shape
        lat = torch.empty(T, H, self.rank + W - self.dim, dtype=q.dtype, device=q.device)
        turn_into(q, lat[..., self.rank :], self.table, positions, self.interleaved)
        head_gemm(q[..., : self.dim], self.up_k, lat[..., : self.rank], transposed=True)
        return head_gemm(attend(lat), self.up_v, out, gate=gate)


def latent_decode(L: Latent, q, cache, block_table, positions, page_size, max_context, gate, out):
    """One query token per request (static shapes, nothing read on the host)."""
    attend = lambda lat: latent_rows(lat, cache, L.rank, block_table, None, positions, page_size, L.scale, max_context)  # noqa: E731
    return L.absorbed(q, positions, attend, gate, out)


def expands(L: Latent, q, page_size: int) -> bool:
    """The expanded form has a kernel for these sizes."""
    r = q.shape[2] - L.dim
    return (q.is_cuda and q.dtype == torch.bfloat16 and L.dim <= 128 and L.vdim <= 128 and r <= 64 and page_size in (16, 32, 64, 128)
            and all(n % 8 == 0 for n in (L.dim, L.vdim, r, L.rank)))  # fmt: skip


def latent_extend(L: Latent, q, cache, batch: wa.ExtendBatch, gate, out):
    """Packed rows of an extend pass: requests with at least ``EXPAND_FROM`` new tokens in the expanded form, the others in the
    absorbed one. ``q`` [T, H, D + r] (not yet rotated), ``gate`` None or [T, H, DV], ``out`` [T, H, DV]."""
    T, ps = q.shape[0], batch.page_size
    long = [r for r, n in enumerate(batch.counts) if n >= EXPAND_FROM] if expands(L, q, ps) else []
    short = [r for r in range(len(batch.counts)) if r not in set(long)]
    longest = max(s + n for s, n in zip(batch.starts, batch.counts))
    if short:
        rows = None
        if long:
            rows = batch.rows_of(tuple(short))
        pick = lambda x: x if rows is None or x is None else x.index_select(0, rows)  # noqa: E731
        req, pos = pick(batch.row_req), pick(batch.positions)
        attend = lambda lat: latent_rows(lat, cache, L.rank, batch.block_table, req, pos, ps, L.scale, longest)  # noqa: E731
        if rows is None:
            return L.absorbed(q, pos, attend, gate, out)
        part = torch.empty(rows.numel(), L.heads, L.vdim, dtype=q.dtype, device=q.device)
        out.index_copy_(0, rows.long(), L.absorbed(pick(q), pos, attend, pick(gate), part))
    pages, table, tiles = batch.expansion(tuple(long))
    ctx = cache.view(-1, ps, cache.shape[2]).index_select(0, pages).view(-1, cache.shape[2])  # the contexts' pages, back to back
    from slime_b200 import ops

    kv = ops.gemm(ctx[:, : L.rank], L.up_kv)
    turn_into(q, q[..., L.dim :], L.table, batch.positions, L.interleaved)
    flat = lambda x: None if x is None else x.flatten(1)  # noqa: E731
    rule = wa.Rule.of(q, L.vdim, L.scale, gate=flat(gate))
    D, DV, r = L.dim, L.vdim, q.shape[2] - L.dim
    assert q.stride(1) == D + r and q.stride(2) == 1 and out.stride(1) == DV
    rc = _lib.lib().sb_flash_latent(
        P(q), P(kv), P(ctx[:, L.rank :]), P(kv[:, L.heads * D :]), P(table), P(tiles), P(out), tiles.shape[0], T, L.heads, D, r, DV, ps,
        table.stride(0), ctx.shape[0], q.stride(0), kv.stride(0), ctx.stride(0), kv.stride(0), out.stride(0), ctypes.byref(rule),
        P(_lib.status_word(q.device)), _lib.stream(),
    )  # fmt: skip
    _lib.check(rc, "sb_flash_latent")
    return out

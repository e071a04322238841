"""Attention over the paged KV cache, for prompts (``window_extend``) and single tokens (``window_decode``).

A query at position i sees key j when ``j <= i`` and (``j`` is in its window, ``i - j < window``, and in its chunk, ``j // chunk ==
i // chunk``; or ``j < keep_first``). Its score is ``scale * q.k``, capped to ``softcap * tanh(score / softcap)``, plus
``bias[i - j, head]`` (``bias`` [N, Hq] fp32 by distance, the last row for everything beyond), minus ``slope[head] * (i - j)``; None:
no such term. ``sinks`` [Hq]: score of an extra softmax column
without a value (None: no such column). The output is multiplied by ``out_scale`` and by ``sigmoid(gate)`` (``gate``: [T, Hq] logits, or
[T, Hq * DV]); ``out`` may be a column range of a wider matrix. Keys and values are read from the cache only,
so a prompt's later portions, portions of several requests and single tokens beside them are one launch.

``pair``: query heads 2 i and 2 i + 1 are two attentions over the same values, of which output head i is the normed difference
(``Pair``); the output then has half as many heads as the queries.

Dispatch on CUDA: bf16 with head widths that are multiples of 8 up to 128 run on the tensor cores
(``csrc/flash_window_sm100.cu``, ``csrc/decode_attn_sm100.cu``), everything else, fp32 included, on the CUDA-core kernel
``csrc/window_attn.cu``. CPU tensors run the definition below.
"""

from __future__ import annotations

import ctypes
import dataclasses

import numpy as np
import torch

from slime_b200.ops import _checks, _lib

P = _lib.ptr
NO_WINDOW = 2**31 - 1
TILE = 128  # query rows (tokens x heads of one kv head) and keys per tile of the tensor-core kernels


def tile_tokens(heads: int, kv_heads: int) -> int:
    """Query tokens of one tile: the heads that share a kv head are stacked into the tile's rows."""
    return TILE // (heads // kv_heads) if heads // kv_heads <= TILE else 0


@dataclasses.dataclass
class ExtendBatch:
    """Where the packed new tokens of a pass stand: row t belongs to request ``row_req[t]`` at position ``positions[t]``;
    request r's pages are ``block_table[r]``. ``starts`` / ``counts`` (host): first position and number of new tokens of
    every request, from which the query tiles of a launch are cut. ``state_slots`` (host): slot of every request's recurrent
    state, for models that have one."""

    block_table: torch.Tensor  # [requests, pages] int32
    row_req: torch.Tensor  # [T] int32
    positions: torch.Tensor  # [T] int32
    starts: list[int]
    counts: list[int]
    page_size: int
    state_slots: list[int] | None = None
    pages: list[list[int]] | None = None  # the same as block_table, on the host
    _tiles: dict = dataclasses.field(default_factory=dict)

    @classmethod
    def build(cls, pages: list[list[int]], starts, counts, page_size: int, device, upload=None, state_slots=None):
        """``upload(ndarray) -> int32 device tensor``; default: a plain copy."""
        up = upload or (lambda a: torch.from_numpy(np.ascontiguousarray(a, dtype=np.int32)).to(device))
        width = max(len(p) for p in pages)
        table = np.zeros((len(pages), width), dtype=np.int32)
        for r, p in enumerate(pages):
            table[r, : len(p)] = p
        req = np.repeat(np.arange(len(pages)), counts)
        pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, counts)])
        return cls(up(table), up(req), up(pos), [int(s) for s in starts], [int(n) for n in counts], page_size,
                   state_slots, pages)

    def tiles(self, tokens: int, requests: tuple[int, ...] | None = None) -> torch.Tensor:
        """[n, 4] int32 (first row, tokens, first position, request) of query tiles of at most ``tokens`` tokens (of some requests
        only)."""

        def make():
            rows, first = [], np.concatenate([[0], np.cumsum(self.counts)])
            for r in range(len(self.counts)) if requests is None else requests:
                off = np.arange(0, self.counts[r], tokens)
                rows.append(np.stack([first[r] + off, np.minimum(tokens, self.counts[r] - off), self.starts[r] + off, np.full_like(off, r)], 1))
            return np.concatenate(rows)

        return self._cached((tokens, requests), make)

    def _cached(self, key, make):
        """``make() -> ndarray`` as an int32 device tensor, built once per pass."""
        if key not in self._tiles:
            host = torch.from_numpy(np.ascontiguousarray(make(), dtype=np.int32))
            if self.row_req.is_cuda:
                host = host.pin_memory()
            self._tiles[key] = host.to(self.row_req.device, non_blocking=True)
        return self._tiles[key]

    def rows_of(self, requests: tuple[int, ...]) -> torch.Tensor:
        """Packed rows of some requests."""
        first = np.concatenate([[0], np.cumsum(self.counts)])
        return self._cached(("rows", requests), lambda: np.concatenate([np.arange(first[r], first[r] + self.counts[r]) for r in requests]))

    def expansion(self, requests: tuple[int, ...], tokens: int = TILE) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
        """For a pass over copies of some requests' contexts, laid page by page behind one another: the pages to copy, the block
        table of the copies [requests, pages] and the query tiles (as ``tiles``, of these requests only)."""
        count = [-(-(self.starts[r] + self.counts[r]) // self.page_size) for r in requests]
        begin = np.concatenate([[0], np.cumsum(count)])

        def table():
            out = np.zeros((len(self.counts), max(count)), dtype=np.int32)
            for r, b, n in zip(requests, begin, count):
                out[r, :n] = np.arange(b, b + n)
            return out

        pages = self._cached(("pages", requests), lambda: np.concatenate([self.pages[r][:n] for r, n in zip(requests, count)]))
        return pages, self._cached(("table", requests), table), self.tiles(tokens, requests)

    def segments(self) -> torch.Tensor:
        """[requests, 4] int32: first row, tokens, first position, state slot."""
        first = np.concatenate([[0], np.cumsum(self.counts)[:-1]])
        return self._cached("segments", lambda: np.stack([first, self.counts, self.starts, self.state_slots], 1))


@dataclasses.dataclass(frozen=True)
class Pair:
    """Output head of two attentions: ``d / sqrt(mean(d^2) + eps) * gain`` with ``d = a1 - weight a2`` (``weight``: fp32 tensor of one
    element)."""

    weight: torch.Tensor
    gain: float
    eps: float


class Rule(ctypes.Structure):
    """``csrc/attn_rule.cuh::AttnRule``: what a query sees and how its scores are made."""

    _fields_ = [(n, ctypes.c_int) for n in ("bytes", "window", "keep_first", "chunk")] + [
        (n, ctypes.c_float) for n in ("scale", "out_scale", "softcap")] + [(n, ctypes.c_int) for n in ("bias_rows", "gate_width")] + [
        ("pair_gain", ctypes.c_float), ("gate_pitch", ctypes.c_long), ("pair_eps", ctypes.c_float), ("reserved", ctypes.c_int)] + [
        (n, ctypes.c_void_p) for n in ("slopes", "sinks", "bias", "gate", "pair")]  # fmt: skip

    @classmethod
    def of(cls, q, DV, scale, window=None, keep_first=0, slopes=None, sinks=None, out_scale=1.0, chunk=None, softcap=None, bias=None, gate=None,
           pair: Pair | None = None):  # fmt: skip
        T, Hq = q.shape[:2]
        for t in (slopes, sinks, bias):
            assert t is None or (t.dtype == torch.float32 and t.is_contiguous() and t.shape[-1] == Hq)
        width = 0
        if gate is not None:
            width = gate.shape[1] // Hq
            assert gate.dtype == q.dtype and gate.stride(1) == 1 and gate.shape in ((T, Hq), (T, Hq * DV))
        w = None if pair is None else pair.weight
        assert w is None or (w.dtype == torch.float32 and w.numel() == 1)
        return cls(ctypes.sizeof(cls), NO_WINDOW if window is None else int(window), int(keep_first), int(chunk or 0), float(scale),
                   float(out_scale), float(softcap or 0.0), 0 if bias is None else bias.shape[0], width, pair.gain if pair else 1.0,
                   0 if gate is None else gate.stride(0), pair.eps if pair else 0.0, 0, P(slopes), P(sinks), P(bias), P(gate), P(w))  # fmt: skip

    def reach(self, longest: int) -> int:
        """Most keys a query sees of a sequence of ``longest`` tokens."""
        return min(longest, min(self.window, self.chunk or longest, longest) + self.keep_first)


def _reference(q, k_cache, v_cache, table, row_req, positions, page_size, scale, window=None, keep_first=0, slopes=None, sinks=None,
               out_scale=1.0, chunk=None, softcap=None, bias=None, gate=None, pair=None):  # fmt: skip
    T, Hq, _ = q.shape
    Hkv, dv = k_cache.shape[1], v_cache.shape[2]
    out = torch.empty(T, Hq // 2 if pair else Hq, dv, dtype=q.dtype)
    req = torch.arange(T) if row_req is None else row_req.long()
    for r in req.unique().tolist():
        rows = (req == r).nonzero().flatten()
        pos = positions[rows].long()
        j = torch.arange(int(pos.max()) + 1)
        slots = table[r, j // page_size].long() * page_size + j % page_size
        k, v = k_cache[slots].float(), v_cache[slots].float()
        dist = pos[:, None] - j[None, :]
        near = torch.ones_like(dist, dtype=torch.bool) if window is None else dist < window
        if chunk:
            near &= j[None, :] // chunk == pos[:, None] // chunk
        see = (dist >= 0) & (near | (j[None, :] < keep_first))
        qr = q[rows].float().view(len(rows), Hkv, Hq // Hkv, -1)
        s = torch.einsum("tghd,jgd->tghj", qr, k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if bias is not None:
            s = s + bias[dist.clamp(0, bias.shape[0] - 1)].permute(0, 2, 1).reshape(s.shape)
        if slopes is not None:
            s = s - slopes.view(1, Hkv, Hq // Hkv, 1) * dist[:, None, None, :].float()
        s = s.masked_fill(~see[:, None, None, :], float("-inf"))
        if sinks is not None:
            s = torch.cat([s, sinks.view(1, Hkv, Hq // Hkv, 1).expand(len(rows), -1, -1, 1)], -1)
        p = s.softmax(-1)[..., : len(j)] * out_scale
        y = torch.einsum("tghj,jgd->tghd", p, v).reshape(len(rows), Hq, dv)
        if pair is not None:
            y = y[:, 0::2] - pair.weight * y[:, 1::2]
            y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + pair.eps) * pair.gain
        if gate is not None:
            y = y * torch.sigmoid(gate[rows].float()).view(len(rows), Hq, -1)
        out[rows] = y.to(q.dtype)
    return out


def _tensor_core_shape(q, k_cache, v_cache, page_size) -> bool:
    D, DV, G = q.shape[2], v_cache.shape[2], q.shape[1] // k_cache.shape[1]
    return (q.dtype == torch.bfloat16 and D <= 128 and DV <= 128 and D % 8 == 0 and DV % 8 == 0 and G <= TILE and q.stride(0) % 8 == 0
            and page_size in (16, 32, 64, 128))  # fmt: skip


def simt(q, k_cache, v_cache, table, row_req, positions, page_size, rule: Rule, out):
    """The CUDA-core kernel. ``v_cache`` may be the first columns of a cache that keeps one vector per token."""
    T, Hq, D = q.shape
    assert k_cache.is_contiguous() and v_cache.stride(2) == 1 and v_cache.stride(0) == v_cache.shape[1] * v_cache.stride(1)
    rc = _lib.lib().sb_window_attn(
        P(q), P(k_cache), P(v_cache), P(table), P(row_req), P(positions), P(out), T, Hq, k_cache.shape[1], D, v_cache.shape[2], page_size,
        table.stride(0), q.stride(0), out.stride(0), v_cache.stride(1), ctypes.byref(rule), int(q.dtype == torch.float32), _lib.stream(),
    )  # fmt: skip
    _lib.check(rc, "sb_window_attn")
    return out


def _output(out, T, Hq, DV, q):
    """[T, Hq, DV] view of ``out`` [T, Hq * DV], or a new tensor."""
    if out is None:
        return torch.empty(T, Hq, DV, dtype=q.dtype, device=q.device)
    assert out.dtype == q.dtype and out.stride(1) == 1 and out.shape == (T, Hq * DV)
    return out.unflatten(1, (Hq, DV))


def _into(out, res):
    return res if out is None else out.copy_(res.flatten(1)).unflatten(1, res.shape[1:])


def window_extend(q, k_cache, v_cache, batch: ExtendBatch, scale, window=None, keep_first=0, slopes=None, sinks=None, out_scale=1.0,
                  out=None, *, chunk=None, softcap=None, bias=None, gate=None, pair=None):  # fmt: skip
    """Attention of the packed rows ``q`` [T, Hq, D] (a strided view is fine) -> [T, Hq, DV]. The rows' own keys and values
    must already be in the cache."""
    T, Hq, D = q.shape
    Hkv, DV = k_cache.shape[1], v_cache.shape[2]
    form = (scale, window, keep_first, slopes, sinks, out_scale, chunk, softcap, bias, gate, pair)
    _checks.index_range("window_extend", "block_table", batch.block_table, upper=k_cache.shape[0] // batch.page_size)
    if not q.is_cuda:
        return _into(out, _reference(q, k_cache, v_cache, batch.block_table, batch.row_req, batch.positions, batch.page_size, *form))
    assert q.stride(2) == 1 and q.stride(1) == D and k_cache.is_contiguous() and v_cache.is_contiguous()
    out, rule = _output(out, T, Hq // 2 if pair else Hq, DV, q), Rule.of(q, DV, *form)
    if _tensor_core_shape(q, k_cache, v_cache, batch.page_size):
        tiles = batch.tiles(tile_tokens(Hq, Hkv))
        rc = _lib.lib().sb_flash_window(
            P(q), P(k_cache), P(v_cache), P(batch.block_table), P(tiles), P(out), tiles.shape[0], T, Hq, Hkv, D, DV, batch.page_size,
            batch.block_table.stride(0), k_cache.shape[0], q.stride(0), out.stride(0), ctypes.byref(rule), P(_lib.status_word(q.device)),
            _lib.stream(),
        )  # fmt: skip
        if rc != -1:  # -1: an alignment the kernel does not take
            _lib.check(rc, "sb_flash_window")
            return out
    return simt(q, k_cache, v_cache, batch.block_table, batch.row_req, batch.positions, batch.page_size, rule, out)


def decode_splits(rows: int, groups: int, reach: int, device, resident: int = 2, tile: int = TILE, limit: int = 16) -> int:
    """Key ranges of one query's launch over ``reach`` keys in tiles of ``tile``: enough CTAs for the machine (``resident`` on an SM), no
    more than the tiles or ``limit``."""
    from slime_b200 import ops

    tiles = -(-reach // tile) + 1  # a window rarely starts at a tile's edge
    most = -(-tiles // 16)  # ranges of 16 tiles: what a launch that must not look at the batch takes
    if ops.BATCH_INVARIANT:
        splits = most
    else:  # a CTA that has an SM to itself walks a longer range rather than wait for a second turn
        splits = max(most if resident > 1 else 1, (resident * _lib.sm_count(device)) // max(rows * groups, 1))
    return max(1, min(limit, splits, tiles))


def window_decode(q, k_cache, v_cache, block_table, seq_lens, positions, page_size, scale, window=None, keep_first=0, slopes=None,
                  max_context: int | None = None, sinks=None, out_scale=1.0, out=None, *, chunk=None, softcap=None, bias=None, gate=None,
                  pair=None):  # fmt: skip
    """One query token per request: ``q`` [B, Hq, D] at ``positions`` = ``seq_lens - 1``, pages in ``block_table`` [B, W].
    Static shapes, nothing read on the host (``max_context``: upper bound of the lengths, from which the number of splits
    follows)."""
    B, Hq, D = q.shape
    Hkv, DV = k_cache.shape[1], v_cache.shape[2]
    form = (scale, window, keep_first, slopes, sinks, out_scale, chunk, softcap, bias, gate, pair)
    if _checks.enabled():
        _checks.paged("window_decode", block_table, seq_lens, page_size, k_cache.shape[0])
    if not q.is_cuda:
        return _into(out, _reference(q, k_cache, v_cache, block_table, None, positions, page_size, *form))
    assert q.stride(2) == 1 and q.stride(1) == D and k_cache.is_contiguous() and v_cache.is_contiguous()
    out, rule = _output(out, B, Hq // 2 if pair else Hq, DV, q), Rule.of(q, DV, *form)
    if _tensor_core_shape(q, k_cache, v_cache, page_size) and Hq // Hkv <= 16:
        longest = min(max_context or block_table.shape[1] * page_size, block_table.shape[1] * page_size)
        splits = decode_splits(B, Hkv, rule.reach(longest), q.device)
        wd = 64 if max(D, DV) <= 64 else 128
        part = torch.empty(B * Hq * splits * (wd + 2), dtype=torch.float32, device=q.device) if splits > 1 else None
        ml = part[B * Hq * splits * wd :] if splits > 1 else None
        rc = _lib.lib().sb_paged_decode_window(
            P(q), P(k_cache), P(v_cache), P(block_table), P(seq_lens), P(out), P(part), P(ml), B, Hq, Hkv, D, DV, page_size,
            block_table.stride(0), k_cache.shape[0], q.stride(0), out.stride(0), splits, ctypes.byref(rule), P(_lib.status_word(q.device)),
            _lib.stream(),
        )  # fmt: skip
        if rc != -1:
            _lib.check(rc, "sb_paged_decode_window")
            return out
    return simt(q, k_cache, v_cache, block_table, None, positions, page_size, rule, out)

"""Where the matrices of a specified layer (``models/layer_spec.py``) lie in the engine's fused buffers.

Everything that reads a layer's normed input is one matrix ``in`` (rows: the projections of all its mixers, and of the
feed-forward when it runs beside them), everything that ends in the residual stream is one matrix ``out`` (columns: the
mixers' heads, the feed-forward's hidden units). So a layer costs two large products whatever it is made of, the products'
sum over mixers and feed-forward is the second one's inner product, and one all-reduce covers it. Two-factor projections
share a third, block-diagonal matrix ``low`` that reads a column range of the first product.

Latent attention's down-projections are rows of ``in``; the expansions of its latents stay matrices of their own
(``up_q``, ``up_kv``). A mixture beside the mixer contributes its shared expert to ``in`` and ``out`` as a dense feed-forward does.

A checkpoint tensor that holds several projections behind one another (Mamba-2's input projection) is taken apart into ranges
of its own (``LayerProjections.split``), so that every rank has the heads it computes.

Every range starts at a multiple of 8 (16 bytes in bf16); what is in between is zero in the matrices.
"""

from __future__ import annotations

from slime_b200.models.layer_spec import DeltaSpec, LatentSpec, LayerSpec, MatrixMemorySpec, StateSpaceSpec


def up8(n: int) -> int:
    return -(-n // 8) * 8


class LayerProjections:
    """``ins[name] = (first row, rows)`` and ``outs[name] = (first column, columns)`` of this rank's part of checkpoint tensor
    ``name`` (behind ``l<i>.``); ``whole``: names that every rank holds completely; ``biased``: names with a bias (tensor
    ``<name>.b``); ``out_biased``: the output projections that have one. ``split[name]``: the ranges (names in ``ins``) a checkpoint tensor is made
    of, with their rows there. ``ff``: (first row, width per rank) of the dense feed-forward in ``in``, or None. ``low[prefix]``: the second factors of mixer
    ``prefix``: (first column in the first product, inner width, rows, {name: (first row, rows, first column, columns)})."""

    def __init__(self, spec: LayerSpec, tp: int = 1):
        self.spec, self.tp = spec, tp
        self.ins: dict[str, tuple[int, int]] = {}
        self.outs: dict[str, tuple[int, int]] = {}
        self.low: dict[str, tuple[int, int, int, dict]] = {}
        self.whole: set[str] = set()
        self.biased: set[str] = set()
        self.out_biased: set[str] = set()
        self.split: dict[str, list[tuple[str, int]]] = {}
        self.ff: tuple[int, int] | None = None
        self.in_rows = self.out_cols = 0
        for p, m, _ in spec.branches():
            if m.heads % tp or m.kv_heads % tp:
                raise ValueError(f"{m.heads} and {m.kv_heads} heads do not divide over {tp} tensor-parallel ranks")
            h, g = m.heads // tp, m.kv_heads // tp
            if isinstance(m, LatentSpec):
                self._in(p + "dq", m.q_rank)
                self._in(p + "dkv", m.cached)
                self.whole |= {p + "dq", p + "dkv"}
                self._gate(p, m)
            elif isinstance(m, DeltaSpec):
                self._in(p + "q", g * m.dim)
                self._in(p + "k", g * m.dim)
                self._in(p + "v", h * m.vdim)
                self._delta(p, m, h)
            elif isinstance(m, StateSpaceSpec):
                parts = [("z", h * m.vdim), ("x", h * m.vdim), ("B", g * m.dim), ("C", g * m.dim), ("dt", h)]
                for n, rows in parts:
                    self._in(p + n, rows)
                self.split[p + "in"] = [(p + n, rows * tp) for n, rows in parts]
            elif isinstance(m, MatrixMemorySpec):
                for n, rows in (("q", h * m.dim), ("k", h * m.dim), ("v", h * m.vdim), ("g", h * m.vdim), ("i", h), ("f", h)):
                    self._in(p + n, rows)
            else:
                own = m.kv_from is None
                self._in(p + "q", h * m.maps * m.dim)
                if own:
                    self._in(p + "k", g * m.maps * m.dim)
                if own and not m.tied_values:
                    self._in(p + "v", g * m.vdim)
                if m.qk_bias:
                    self.biased |= {p + "q", p + "k"} if own else {p + "q"}
                if m.vo_bias:
                    self.biased |= {p + "v"} if own and not m.tied_values else set()
                    self.out_biased.add(p + "o")
                self._gate(p, m)
            self._out(p + "o", h * m.vdim)
        if spec.joint_ff is not None:
            stem, width = spec.joint_ff
            if width % tp:
                raise ValueError(f"a feed-forward of width {width} does not divide over {tp} tensor-parallel ranks")
            f = width // tp
            self.ff = (self.in_rows, f)
            if spec.mlp.gated:  # gate and up rows without a gap: the activation reads them as one range
                self.ins[stem + ".gate"] = (self.in_rows, f)
                self.ins[stem + ".up"] = (self.in_rows + f, f)
                self.in_rows += up8(2 * f)
            else:
                self._in(stem + ".up", f)
            self._out(stem + ".down", f)

    def _gate(self, p: str, m):
        if m.gate is not None:
            self._in(p + "g", m.gate_rows // self.tp)

    def _in(self, name: str, rows: int):
        self.ins[name] = (self.in_rows, rows)
        self.in_rows += up8(rows)

    def _out(self, name: str, cols: int):
        self.outs[name] = (self.out_cols, cols)
        self.out_cols += up8(cols)

    def _delta(self, p: str, m: DeltaSpec, h: int):
        self._in(p + "b", h)
        pairs = [("a", m.decay_rank, m.decays // self.tp), ("g", m.gate_rank, h * m.vdim)]
        for n, rank, rows in pairs:
            if rank is None:
                self._in(p + n, rows)
        first, inner, total, parts = self.in_rows, 0, 0, {}
        for n, rank, rows in pairs:
            if rank is not None:
                self._in(p + n + "1", rank)
                self.whole.add(p + n + "1")
                parts[p + n + "2"] = (total, rows, inner, rank)
                inner, total = inner + up8(rank), total + up8(rows)
        if parts:
            self.low[p] = (first, inner, total, parts)

    def padded(self, ranges: dict) -> bool:
        return any(n % 8 for _, n in ranges.values())

    # ------------------------------------------------------------------ the checkpoint's side
    def tensors(self, width: int) -> dict[str, tuple[int, ...]]:
        """Shapes of the mixers' tensors (and of a feed-forward beside them) in the checkpoint; tp must be 1."""
        assert self.tp == 1
        joined = {n for parts in self.split.values() for n, _ in parts}
        out = {n: (rows, width) for n, (_, rows) in self.ins.items() if n not in joined}
        out.update({n: (sum(rows for _, rows in parts), width) for n, parts in self.split.items()})
        out.update({n + ".b": (width,) for n in self.out_biased})
        out.update({n: (width, cols) for n, (_, cols) in self.outs.items()})
        for _, _, _, parts in self.low.values():
            out.update({n: (rows, cols) for n, (_, rows, _, cols) in parts.items()})
        out.update({n + ".b": (self.ins[n][1],) for n in self.biased})
        for p, m, _ in self.spec.branches():
            if isinstance(m, DeltaSpec):
                g, h = m.kv_heads * m.dim, m.heads * m.vdim
                out.update({p + "q.conv": (g, m.conv), p + "k.conv": (g, m.conv), p + "v.conv": (h, m.conv), p + "A_log": (m.heads,),
                            p + "dt_bias": (m.decays,), p + "norm": (m.vdim,)})  # fmt: skip
                continue
            if isinstance(m, LatentSpec):
                out.update({p + "dq.norm": (m.q_rank,), p + "dkv.norm": (m.kv_rank,), p + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                            p + "uk": (m.heads * m.dim, m.kv_rank), p + "uv": (m.heads * m.vdim, m.kv_rank)})  # fmt: skip
                continue
            if isinstance(m, StateSpaceSpec):
                out.update({p + "conv": (m.channels, m.conv), p + "conv.b": (m.channels,), p + "norm": (m.heads * m.vdim,)})
                out.update({p + n: (m.heads,) for n in ("A_log", "dt_bias", "D")})
                continue
            if isinstance(m, MatrixMemorySpec):
                out.update({p + "i.b": (m.heads,), p + "f.b": (m.heads,), p + "norm": (m.heads * m.vdim,)})
                continue
            if m.qk_norm:
                nq, nk = m.norm_widths()
                out.update({p + "q.norm": (nq,)} if m.kv_from is not None else {p + "q.norm": (nq,), p + "k.norm": (nk,)})
            if m.diff is not None:
                out.update({p + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
            if m.learned_bias is not None:
                out[p + "rel"] = (m.learned_bias.rows, m.heads)
        return out

"""Linear recurrences of the rollout engine (``csrc/linear_scan.cu``): state-space duality (Mamba-2) and matrix memory (mLSTM) over
states that live in slots.

Per head, S [D, DV] in fp32:  ``S <- f S + w k v^T;  o = S^T q`` with one decay f and one weight w per head and token.

* ``StateSpace``: q, k, v = C, B, x, which passed a causal convolution (with bias) over ``taps`` tokens per channel and silu; B and C are shared by
  groups of heads. ``w = softplus(dt + dt_bias)``, ``f = exp(-exp(A_log) w)``; ``skip v`` is added to the output. Times silu(z), RMS normed
  in parts.
* ``MatrixMemory``: log gates ``i = cap tanh((z_i + b_i) / cap)`` and ``g = logsigmoid(cap tanh((z_f + b_f) / cap))``; a running maximum
  ``m <- max(g + m, i)`` (0 at first) keeps ``f = exp(g + m' - m)`` and ``w = exp(i - m)`` in range; a normaliser ``n <- f n + w k`` beside S; q
  times D^-1/2; the output over ``max(|n.q|, exp(-m)) + 1e-6``, RMS normed per head, times sigmoid(z).

``extend`` takes the packed rows of a pass (portions of prompts, single tokens), ``step`` one token per decode row. Both read and leave a
request's state in its slot. A sequence's first token starts from zeros whatever the slot holds. The recurrence is evaluated token by
token in fp32, so results do not depend on where a prompt was cut.

CUDA tensors run the kernels; CPU tensors run the definitions in this file.
"""

from __future__ import annotations

import dataclasses

import torch

from slime_b200.ops import _checks, _lib

P = _lib.ptr
RUN = 16  # tokens of one run of the token-parallel part


@dataclasses.dataclass
class SlotState:
    """What one recurrent mixer keeps, all slots: ``state`` [slots, H, D, DV]; ``ring`` [slots, taps, channels], the convolution's inputs by
    position modulo taps; ``norm`` [slots, H, D]; ``top`` [slots, H, 2], the running maximum before a position of even / odd number."""

    state: torch.Tensor
    ring: torch.Tensor | None = None
    norm: torch.Tensor | None = None
    top: torch.Tensor | None = None


def part_gate(o, z, w, parts: int, act: str, eps: float, *, gate_first: bool, den=None, scale: float = 1.0, out=None):
    """``o`` [T, parts * W] fp32 (over ``den`` [T, parts]) RMS normed in equal parts, times ``w``, times ``act(z)`` (``gate_first``: before the
    norm). ``act`` "silu" or "sigmoid". Result of z's type (``out``: a column range of a wider matrix)."""
    T = o.shape[0]
    n = o[0].numel() if T else w.numel()
    W = n // parts
    assert n == parts * W == w.numel() and z.shape == (T, n)
    if not o.is_cuda:
        x = o.reshape(T, parts, W)
        x = x if den is None else x / den.view(T, parts, 1)
        gate = torch.sigmoid(z.float())
        gate = (gate * z.float() if act == "silu" else gate).view(T, parts, W)
        x = x * gate if gate_first else x
        x = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float().view(parts, W) * scale
        y = (x if gate_first else x * gate).flatten(1).to(z.dtype)
        return y if out is None else out.copy_(y)
    if out is None:
        out = torch.empty(T, n, dtype=z.dtype, device=z.device)
    assert o.is_contiguous() and z.stride(1) == 1 and out.stride(1) == 1 and w.dtype == z.dtype == out.dtype and w.is_contiguous()
    rc = _lib.lib().sb_part_gate(P(o), P(den), P(z), P(w), P(out), T, parts, W, z.stride(0), out.stride(0), float(eps), float(scale),
                                 int(act == "sigmoid"), int(gate_first), int(z.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_part_gate")
    return out


def _scan(q, k, v, gates, segs, s: SlotState, *, skip=None, den=None, ring_in=()):
    """The recurrence over packed rows on the device -> o [T, H, DV]."""
    T, H, DV = v.shape
    G, D = q.shape[1:]
    out = torch.empty_like(v)
    ins = [*ring_in, None, None, None][:3]
    widths = [0 if x is None else x.shape[1] for x in ins]
    keep = bool(ring_in)
    rc = _lib.lib().sb_linear_scan(
        P(q), P(k), P(v), P(gates), P(skip), P(out), P(s.state), P(s.norm), P(den), P(segs), segs.shape[0], H, G, D, DV,
        P(s.ring) if keep else None, *(P(x) for x in ins), ring_in[0].stride(0) if keep else 0, *widths, s.ring.shape[1] if keep else 0,
        s.ring.element_size() if keep else 0, _lib.stream(),
    )  # fmt: skip
    _lib.check(rc, "sb_linear_scan")
    return out


def _walk(S, f, w, q, k, v):
    """The recurrence of one request: f, w [n, H], q, k [n, H, D], v [n, H, DV] from S [H, D, DV] -> (o [n, H, DV], S)."""
    out = torch.empty_like(v)
    for t in range(v.shape[0]):
        S = f[t][:, None, None] * S + (w[t][:, None] * k[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


@dataclasses.dataclass
class StateSpace:
    """Projections of the new tokens (column ranges of one wider matrix): ``z``, ``x`` [T, H * DV], ``B``, ``C`` [T, G * D], ``dt`` [T, H]; the layer's
    ``conv`` [channels, taps] and ``conv_b`` (channels x, B, C), ``A_log``, ``dt_bias``, ``skip`` [H] fp32, ``norm`` [H * DV] in ``parts``."""

    z: torch.Tensor
    x: torch.Tensor
    B: torch.Tensor
    C: torch.Tensor
    dt: torch.Tensor
    conv: torch.Tensor
    conv_b: torch.Tensor
    A_log: torch.Tensor
    dt_bias: torch.Tensor
    skip: torch.Tensor
    norm: torch.Tensor
    parts: int
    eps: float
    scale: float = 1.0

    def sizes(self, s: SlotState):
        H, D, DV = s.state.shape[1:]
        return H, self.B.shape[1] // D, D, DV, self.conv.shape[1]

    def check(self, s: SlotState):
        H, G, D, DV, taps = self.sizes(s)
        T, ch = self.x.shape[0], H * DV + 2 * G * D
        assert G > 0 and H % G == 0 and self.z.shape == self.x.shape == (T, H * DV) and self.B.shape == self.C.shape == (T, G * D)
        assert self.dt.shape == (T, H) and self.conv.shape == (ch, taps) and self.conv_b.numel() == ch and s.ring.shape[1:] == (taps, ch)
        if self.x.is_cuda:
            rows = (self.z, self.x, self.B, self.C, self.dt)
            assert len({t.stride(0) for t in rows}) == 1 and all(t.stride(1) == 1 for t in rows)
            assert len({t.dtype for t in (*rows, self.conv, self.conv_b, s.ring)}) == 1
            assert all(t.dtype == torch.float32 and t.numel() == H for t in (self.A_log, self.dt_bias, self.skip))
            assert s.state.is_contiguous() and s.ring.is_contiguous() and self.conv.is_contiguous() and s.state.dtype == torch.float32

    def _finish(self, o, out):
        return part_gate(o, self.z, self.norm, self.parts, "silu", self.eps, gate_first=True, scale=self.scale, out=out)

    def _rows(self, rows: slice, start: int, slot: int, s: SlotState):
        """One request's rows, from its slot and back into it -> o [n, H, DV]."""
        H, G, D, DV, taps = self.sizes(s)
        new = torch.cat([t[rows] for t in (self.x, self.B, self.C)], 1)
        n = new.shape[0]
        past = [s.ring[slot, p % taps] if p >= 0 else torch.zeros_like(new[0]) for p in range(start - taps + 1, start)]
        seen = torch.cat([torch.stack(past), new] if past else [new]).float()
        y = sum(seen[t : t + n] * self.conv[:, t].float() for t in range(taps)) + self.conv_b.float()
        y = y * torch.sigmoid(y)
        for p in range(max(start, start + n - taps + 1), start + n):
            s.ring[slot, p % taps] = new[p - start]
        x, B, C = y.split([H * DV, G * D, G * D], 1)
        x, (B, C) = x.reshape(n, H, DV), (t.reshape(n, G, D).repeat_interleave(H // G, 1) for t in (B, C))
        w = torch.nn.functional.softplus(self.dt[rows].float() + self.dt_bias, threshold=1e9)
        f = torch.exp(-self.A_log.exp() * w)
        S = s.state[slot].clone() if start > 0 else torch.zeros_like(s.state[slot])
        o, s.state[slot] = _walk(S, f, w, C, B, x)
        return o + self.skip[:, None] * x

    def extend(self, s: SlotState, batch, out=None):
        self.check(s)
        H, G, D, DV, taps = self.sizes(s)
        T, segs = self.x.shape[0], batch.segments()
        _checks.index_range("StateSpace.extend", "state_slots", segs[:, 3], upper=s.state.shape[0])
        if not self.x.is_cuda:
            o = torch.empty(T, H, DV)
            for row, n, start, slot in segs.tolist():
                o[row : row + n] = self._rows(slice(row, row + n), start, slot, s)
            return self._finish(o, out)
        runs = batch.tiles(RUN)
        new = lambda *sh: torch.empty(*sh, dtype=torch.float32, device=self.x.device)  # noqa: E731
        x, B, C, gates = new(T, H, DV), new(T, G, D), new(T, G, D), new(T, H, 4)
        rc = _lib.lib().sb_ssd_prep(P(self.x), P(self.B), P(self.C), P(self.dt), self.x.stride(0), P(self.conv), P(self.conv_b), P(self.A_log),
                                    P(self.dt_bias), P(s.ring), P(runs), P(segs), runs.shape[0], P(x), P(B), P(C), P(gates), H, G, D, DV, taps,
                                    int(self.x.dtype == torch.float32), _lib.stream())  # fmt: skip
        _lib.check(rc, "sb_ssd_prep")
        return self._finish(_scan(C, B, x, gates, segs, s, skip=self.skip, ring_in=(self.x, self.B, self.C)), out)

    def step(self, s: SlotState, slots, active, positions, out=None):
        """One token per row: row b belongs to state slot ``slots[b]`` and stands at ``positions[b]``; rows with ``active[b]`` 0 touch no state.
        Static shapes, nothing read on the host."""
        self.check(s)
        H, G, D, DV, taps = self.sizes(s)
        n = self.x.shape[0]
        _checks.index_range("StateSpace.step", "slots", slots, upper=s.state.shape[0])
        if not self.x.is_cuda:
            o = torch.zeros(n, H, DV)
            for b in [b for b in range(n) if int(active[b])]:
                o[b] = self._rows(slice(b, b + 1), int(positions[b]), int(slots[b]), s)[0]
            return self._finish(o, out)
        o = torch.empty(n, H, DV, dtype=torch.float32, device=self.x.device)
        rc = _lib.lib().sb_ssd_step(P(self.x), P(self.B), P(self.C), P(self.dt), self.x.stride(0), P(self.conv), P(self.conv_b), P(self.A_log),
                                    P(self.dt_bias), P(self.skip), P(s.ring), P(s.state), P(slots), P(active), P(positions), P(o), n, H, G, D, DV,
                                    taps, int(self.x.dtype == torch.float32), _lib.stream())  # fmt: skip
        _lib.check(rc, "sb_ssd_step")
        return self._finish(o, out)


@dataclasses.dataclass
class MatrixMemory:
    """Projections of the new tokens (column ranges of one wider matrix): ``q``, ``k`` [T, H * D], ``v``, ``z`` [T, H * DV], ``i``, ``f`` [T, H]; the
    layer's gate biases ``i_b``, ``f_b`` [H] fp32 and ``norm`` [H * DV]."""

    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    i: torch.Tensor
    f: torch.Tensor
    z: torch.Tensor
    i_b: torch.Tensor
    f_b: torch.Tensor
    norm: torch.Tensor
    cap: float
    eps: float
    scale: float = 1.0

    def check(self, s: SlotState):
        H, D, DV = s.state.shape[1:]
        T = self.q.shape[0]
        assert self.q.shape == self.k.shape == (T, H * D) and self.v.shape == self.z.shape == (T, H * DV) and self.i.shape == self.f.shape == (T, H)
        assert s.norm.shape[1:] == (H, D) and s.top.shape[1:] == (H, 2)
        if self.q.is_cuda:
            rows = (self.q, self.k, self.v, self.i, self.f, self.z)
            assert len({t.stride(0) for t in rows}) == 1 and all(t.stride(1) == 1 for t in rows) and len({t.dtype for t in rows}) == 1
            assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (s.state, s.norm, s.top, self.i_b, self.f_b))

    def _finish(self, o, den, out):
        return part_gate(o, self.z, self.norm, o.shape[1], "sigmoid", self.eps, gate_first=False, den=den, scale=self.scale, out=out)

    def _rows(self, rows: slice, start: int, slot: int, s: SlotState):
        """One request's rows, from its slot and back into it -> (o [n, H, DV], divisors [n, H])."""
        H, D, DV = s.state.shape[1:]
        soft = lambda z: self.cap * torch.tanh(z / self.cap)  # noqa: E731
        i = soft(self.i[rows].float() + self.i_b)
        g = torch.nn.functional.logsigmoid(soft(self.f[rows].float() + self.f_b))
        q, k, v = (t[rows].float().reshape(i.shape[0], H, -1) for t in (self.q, self.k, self.v))
        m = s.top[slot, :, start % 2] if start > 0 else torch.zeros(H)
        f, w, least = torch.empty_like(i), torch.empty_like(i), torch.empty_like(i)
        for t in range(i.shape[0]):
            now = torch.maximum(g[t] + m, i[t])
            f[t], w[t], least[t], m = torch.exp(g[t] + m - now), torch.exp(i[t] - now), torch.exp(-now), now
        s.top[slot, :, (start + i.shape[0]) % 2] = m
        both = torch.cat([s.state[slot], s.norm[slot][:, :, None]], -1)  # the normaliser is a column whose v is 1
        o, both = _walk(both if start > 0 else torch.zeros_like(both), f, w, q * D**-0.5, k, torch.cat([v, torch.ones_like(v[..., :1])], -1))
        s.state[slot], s.norm[slot] = both[..., :DV], both[..., DV]
        return o[..., :DV], torch.maximum(o[..., DV].abs(), least) + 1e-6

    def extend(self, s: SlotState, batch, out=None):
        self.check(s)
        H, D, DV = s.state.shape[1:]
        T, segs = self.q.shape[0], batch.segments()
        _checks.index_range("MatrixMemory.extend", "state_slots", segs[:, 3], upper=s.state.shape[0])
        new = lambda *sh: torch.empty(*sh, dtype=torch.float32, device=self.q.device)  # noqa: E731
        den = new(T, H)
        if not self.q.is_cuda:
            o = new(T, H, DV)
            for row, n, start, slot in segs.tolist():
                o[row : row + n], den[row : row + n] = self._rows(slice(row, row + n), start, slot, s)
            return self._finish(o, den, out)
        q, k, v, gates = new(T, H, D), new(T, H, D), new(T, H, DV), new(T, H, 4)
        rc = _lib.lib().sb_memory_prep(P(self.q), P(self.k), P(self.v), P(self.i), P(self.f), self.q.stride(0), P(self.i_b), P(self.f_b), P(s.top),
                                       P(segs), segs.shape[0], T, P(q), P(k), P(v), P(gates), H, D, DV, float(self.cap),
                                       int(self.q.dtype == torch.float32), _lib.stream())  # fmt: skip
        _lib.check(rc, "sb_memory_prep")
        return self._finish(_scan(q, k, v, gates, segs, s, den=den), den, out)

    def step(self, s: SlotState, slots, active, positions, out=None):
        """As ``StateSpace.step``."""
        self.check(s)
        H, D, DV = s.state.shape[1:]
        n = self.q.shape[0]
        _checks.index_range("MatrixMemory.step", "slots", slots, upper=s.state.shape[0])
        o, den = (torch.empty(*sh, dtype=torch.float32, device=self.q.device) for sh in ((n, H, DV), (n, H)))
        if not self.q.is_cuda:
            o.zero_()
            den.fill_(1.0)
            for b in [b for b in range(n) if int(active[b])]:
                o[b : b + 1], den[b : b + 1] = self._rows(slice(b, b + 1), int(positions[b]), int(slots[b]), s)
            return self._finish(o, den, out)
        rc = _lib.lib().sb_memory_step(P(self.q), P(self.k), P(self.v), P(self.i), P(self.f), self.q.stride(0), P(self.i_b), P(self.f_b), P(s.top),
                                       P(s.state), P(s.norm), P(slots), P(active), P(positions), P(o), P(den), n, H, D, DV, float(self.cap),
                                       int(self.q.dtype == torch.float32), _lib.stream())  # fmt: skip
        _lib.check(rc, "sb_memory_step")
        return self._finish(o, den, out)

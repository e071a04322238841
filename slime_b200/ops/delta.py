"""Gated delta rule of the rollout engine (``csrc/delta_rule.cu``): convolution, unit vectors, gates, recurrence over states that
live in slots, output norm and gate.

Per head, S [D, DV] in fp32:  ``S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q``. q, k, v are projections that passed a
causal convolution over ``taps`` tokens per channel and silu; q and k are made unit vectors, q also times D^-1/2.
``g = exp(-exp(A_log) softplus(a + dt_bias))`` per head or per key channel, ``beta = sigmoid(b)``.

``delta_extend`` takes the packed rows of a pass (portions of prompts, single tokens), ``delta_step`` one token per decode row.
Both read and leave a request's state in its slot: ``state`` [slots, H, D, DV] fp32 and ``ring`` [slots, taps, channels], the
convolution's inputs by position modulo taps. A sequence's first token starts from zeros whatever the slot holds. The
recurrence is evaluated token by token, so results do not depend on where a prompt was cut.

CUDA tensors run the kernels; CPU tensors run the definitions in this file.
"""

from __future__ import annotations

import dataclasses

import torch

from slime_b200.ops import _checks, _lib

P = _lib.ptr
RUN = 16  # tokens of one warp's run in the token-parallel part


@dataclasses.dataclass
class DeltaInputs:
    """Projections of the new tokens (column ranges of wider matrices are fine; q, k, v with one row pitch): ``q``, ``k`` [T, G * D],
    ``v`` [T, H * DV], ``a`` [T, H] or [T, H * D] (decay per head or per key channel), ``b`` [T, H]; the layer's ``conv``
    [2 G D + H DV, taps] (channels q, k, v), ``A_log`` [H] and ``dt_bias`` fp32."""

    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    a: torch.Tensor
    b: torch.Tensor
    conv: torch.Tensor
    A_log: torch.Tensor
    dt_bias: torch.Tensor

    def gated(self, z, w, act: str, eps: float, scale: float = 1.0) -> "DeltaMixer":
        return DeltaMixer(self, z, w, act, eps, scale)

    def sizes(self, state):
        """(H, G, D, DV, taps, per_channel)"""
        H, D, DV = state.shape[1:]
        return H, self.q.shape[1] // D, D, DV, self.conv.shape[1], self.a.shape[1] != H

    def check(self, state, ring):
        H, G, D, DV, taps, pc = self.sizes(state)
        T = self.q.shape[0]
        C = 2 * G * D + H * DV
        assert H % G == 0 and self.k.shape == self.q.shape == (T, G * D) and self.v.shape == (T, H * DV)
        assert self.a.shape == (T, H * D if pc else H) and self.b.shape == (T, H) and self.dt_bias.numel() == self.a.shape[1]
        assert self.conv.shape == (C, taps) and ring.shape[1:] == (taps, C) and self.A_log.numel() == H
        if self.q.is_cuda:
            assert self.q.stride(0) == self.k.stride(0) == self.v.stride(0) and all(x.stride(1) == 1 for x in (self.q, self.k, self.v, self.a, self.b))
            assert len({x.dtype for x in (self.q, self.k, self.v, self.a, self.b, self.conv, ring)}) == 1
            assert state.dtype == self.A_log.dtype == self.dt_bias.dtype == torch.float32
            assert state.is_contiguous() and ring.is_contiguous() and self.conv.is_contiguous()


def _decay(x: DeltaInputs, H, D, per_channel):
    """[T, H, D]"""
    z = torch.nn.functional.softplus(x.a.float() + x.dt_bias.float(), threshold=1e9)
    z = z.view(-1, H, D) if per_channel else z[:, :, None].expand(-1, -1, D)
    return torch.exp(-x.A_log.float().exp()[None, :, None] * z)


def _unit(x):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def _reference_rows(x: DeltaInputs, rows: slice, start: int, slot: int, state, ring):
    """One request's rows, from its slot and back into it -> o [n, H, DV]."""
    H, G, D, DV, taps, pc = x.sizes(state)
    new = torch.cat([t[rows] for t in (x.q, x.k, x.v)], 1)
    n = new.shape[0]
    past = torch.stack([ring[slot, p % taps] if p >= 0 else torch.zeros_like(new[0]) for p in range(start - taps + 1, start)]) if taps > 1 else new[:0]
    seen = torch.cat([past, new]).float()  # positions start - taps + 1 ...
    y = sum(seen[s : s + n] * x.conv[:, s].float() for s in range(taps))
    y = y * torch.sigmoid(y)
    for p in range(max(start, start + n - taps + 1), start + n):
        ring[slot, p % taps] = new[p - start]
    q, k, v = y.split([G * D, G * D, H * DV], 1)
    q, k = (_unit(t.view(n, G, D)).repeat_interleave(H // G, 1) for t in (q, k))
    q, v = q * D**-0.5, v.view(n, H, DV)
    part = dataclasses.replace(x, a=x.a[rows])
    g, beta = _decay(part, H, D, pc), torch.sigmoid(x.b[rows].float())
    S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
    out = torch.empty(n, H, DV)
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    state[slot] = S
    return out


def delta_extend(x: DeltaInputs, state, ring, batch) -> torch.Tensor:
    """Recurrence over the packed rows of ``batch`` (``window_attention.ExtendBatch`` with state slots) -> o [T, H, DV] fp32."""
    x.check(state, ring)
    H, G, D, DV, taps, pc = x.sizes(state)
    T = x.q.shape[0]
    segs = batch.segments()
    _checks.index_range("delta_extend", "state_slots", segs[:, 3], upper=state.shape[0])
    if not x.q.is_cuda:
        out = torch.empty(T, H, DV)
        for row, n, start, slot in segs.tolist():
            out[row : row + n] = _reference_rows(x, slice(row, row + n), start, slot, state, ring)
        return out
    runs = batch.tiles(RUN)
    f32, lib = int(x.q.dtype == torch.float32), _lib.lib()
    new = lambda *s: torch.empty(*s, dtype=torch.float32, device=x.q.device)  # noqa: E731
    q, k, v, beta, qk, out = new(T, G, D), new(T, G, D), new(T, H, DV), new(T, H), new(T, G), new(T, H, DV)
    g = new(T, H, D) if pc else new(T, H)
    rc = lib.sb_delta_prep(P(x.q), P(x.k), P(x.v), P(x.a), P(x.b), x.q.stride(0), x.a.stride(0), x.b.stride(0), P(x.conv), P(x.A_log),
                           P(x.dt_bias), P(ring), P(runs), P(segs), runs.shape[0], P(q), P(k), P(v), P(g), P(beta), P(qk), H, G, D, DV, taps,
                           int(pc), f32, _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_delta_prep")
    rc = lib.sb_delta_scan(P(x.q), P(x.k), P(x.v), x.q.stride(0), P(ring), P(state), P(segs), segs.shape[0], P(q), P(k), P(v), P(g), P(beta),
                           P(qk), P(out), H, G, D, DV, taps, int(pc), f32, _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_delta_scan")
    return out


def head_gate(o, z, w, act: str, eps: float, scale: float = 1.0, out=None):
    """``scale * o / rms(o) * w * act(z)`` per head: ``o`` [T, H, DV] fp32, ``z`` [T, H * DV], ``w`` [DV] shared by the heads; ``act``
    "silu" or "sigmoid". Result [T, H * DV] of z's type (``out``: a column range of a wider matrix)."""
    T, H, DV = o.shape
    if not o.is_cuda:
        gate = torch.sigmoid(z.float())
        gate = gate * z.float() if act == "silu" else gate
        y = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w.float() * gate.view(T, H, DV) * scale
        y = y.flatten(1).to(z.dtype)
        return y if out is None else out.copy_(y)
    if out is None:
        out = torch.empty(T, H * DV, dtype=z.dtype, device=z.device)
    assert o.is_contiguous() and z.stride(1) == 1 and out.stride(1) == 1 and w.dtype == z.dtype == out.dtype
    rc = _lib.lib().sb_head_gate(P(o), P(z), P(w), P(out), T, H, DV, z.stride(0), out.stride(0), float(eps), float(scale), int(act == "sigmoid"),
                                 int(z.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_head_gate")
    return out


def delta_step(x: DeltaInputs, state, ring, slots, active, positions, z, w, act: str, eps: float, scale: float = 1.0, out=None):
    """One token per row: row b belongs to state slot ``slots[b]`` and stands at ``positions[b]``; rows with ``active[b]`` 0 touch no
    state and give zeros. Includes ``head_gate``. Static shapes, nothing read on the host."""
    x.check(state, ring)
    H, G, D, DV, taps, pc = x.sizes(state)
    B = x.q.shape[0]
    _checks.index_range("delta_step", "slots", slots, upper=state.shape[0])
    if not x.q.is_cuda:
        o = torch.zeros(B, H, DV)
        live = [b for b in range(B) if int(active[b])]
        for b in live:
            o[b] = _reference_rows(x, slice(b, b + 1), int(positions[b]), int(slots[b]), state, ring)[0]
        return head_gate(o, z, w, act, eps, scale, out)
    if out is None:
        out = torch.empty(B, H * DV, dtype=z.dtype, device=z.device)
    assert z.stride(1) == 1 and out.stride(1) == 1 and w.dtype == z.dtype == out.dtype == x.q.dtype
    rc = _lib.lib().sb_delta_step(P(x.q), P(x.k), P(x.v), P(x.a), P(x.b), x.q.stride(0), x.a.stride(0), x.b.stride(0), P(x.conv), P(x.A_log),
                                  P(x.dt_bias), P(ring), P(state), P(slots), P(active), P(positions), P(z), P(w), P(out), z.stride(0),
                                  out.stride(0), float(eps), float(scale), int(act == "sigmoid"), B, H, G, D, DV, taps, int(pc),
                                  int(x.q.dtype == torch.float32), _lib.stream())  # fmt: skip
    _lib.check(rc, "sb_delta_step")
    return out


@dataclasses.dataclass
class DeltaMixer:
    """The rule with the norm and gate of its output (``head_gate``), as the engine runs recurrent mixers: ``extend`` over the packed rows of a
    pass, ``step`` over the decode rows, both on the slots of a ``SlotState``."""

    inputs: DeltaInputs
    z: torch.Tensor
    w: torch.Tensor
    act: str
    eps: float
    scale: float = 1.0

    def extend(self, s, batch, out=None):
        return head_gate(delta_extend(self.inputs, s.state, s.ring, batch), self.z, self.w, self.act, self.eps, self.scale, out)

    def step(self, s, slots, active, positions, out=None):
        return delta_step(self.inputs, s.state, s.ring, slots, active, positions, self.z, self.w, self.act, self.eps, self.scale, out)

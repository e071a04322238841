"""Plain, slow definition of the Pebodra decoder, one function per mechanism, float64 by default.

No batching, no cache: every function takes one whole sequence and writes the equation down. It shares no code with the
product path and is what the tests of that path are compared with.
"""

from __future__ import annotations

import torch


def rms_parts(x, parts, eps):
    """Every one of ``parts`` equal pieces of a row over its own root mean square."""
    p = x.unflatten(-1, (parts, -1))
    return (p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)).flatten(-2)


def silu(z):
    return z * torch.sigmoid(z)


def rotate_halves(x, dims, base):
    """x [T, heads, d] of positions 0..T-1: coordinates (i, i + dims / 2) of the first ``dims`` turned by position * base^(-2i / dims)."""
    half, out = dims // 2, x.clone()
    freq = torch.tensor([base ** (-2 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * freq
    c, s = angle.cos(), angle.sin()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half], out[..., half:dims] = u * c - v * s, v * c + u * s
    return out


def window_mask(T, size):
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size)


def pair_weight(lq1, lk1, lq2, lk2, diff):
    """Factor of the second map."""
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def pair_attention(q, k, v, scale, see, weight, diff, eps):
    """Difference of two attentions over the same values: q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv], see [T, T] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        maps = [torch.softmax(((q[:, h, m] @ k[:, g, m].t()) * scale).masked_fill(~see, float("-inf")), -1) @ v[:, g] for m in (0, 1)]
        out.append(rms_parts(maps[0] - weight * maps[1], 1, eps) * (1 - diff))
    return torch.stack(out, 1)


def attention_keys(h, W, m, eps):
    """Keys and values as layers may share them."""
    T, G, d = h.shape[0], m["kv_heads"], m["dim"]
    k = rms_parts((h @ W("k").t() + W("k.b")).view(T, G * 2, d), 1, eps) * W("k.norm")
    return rotate_halves(k, m["rot"]["dims"], m["rot"]["base"]).view(T, G, 2, d), (h @ W("v").t() + W("v.b")).view(T, G, -1)


def attention(h, W, m, eps, kv):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    q = rms_parts((h @ W("q").t() + W("q.b")).view(T, H * 2, d), 1, eps) * W("q.norm")
    q = rotate_halves(q, m["rot"]["dims"], m["rot"]["base"]).view(T, H, 2, d)
    weight = pair_weight(W("lq1"), W("lk1"), W("lq2"), W("lk2"), m["diff"])
    y = pair_attention(q, *kv, m["scale"], window_mask(T, m["mask"]["size"]), weight, m["diff"], eps)
    return y.reshape(T, -1) @ W("o").t() + W("o.b")


def short_conv(x, w, b):
    """Causal convolution of every channel over its last taps, silu."""
    T, taps = x.shape[0], w.shape[1]
    past = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return silu(sum(past[s : s + T] * w[:, s] for s in range(taps)) + b)


def state_space(x, B, C, step, rate, skip):
    """S <- exp(-rate step) S + step B x^T, y = S^T C + skip x per head: x [T, H, dv], B / C [T, G, n], step [T, H], rate / skip [H]."""
    T, H, dv = x.shape
    G, n = B.shape[1:]
    out = torch.empty_like(x)
    for h in range(H):
        g, S = h // (H // G), x.new_zeros(n, dv)
        for t in range(T):
            S = torch.exp(-rate[h] * step[t, h]) * S + step[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S.t() @ C[t, g] + skip[h] * x[t, h]
    return out


def mamba2(h, W, m, eps):
    T, H, dv, n, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    z, x, B, C, dt = (h @ W("in").t()).split([H * dv, H * dv, G * n, G * n, H], 1)
    x, B, C = short_conv(torch.cat([x, B, C], 1), W("conv"), W("conv.b")).split([H * dv, G * n, G * n], 1)
    step = dt + W("dt_bias")
    step = torch.clamp(step, min=0) + torch.log1p(torch.exp(-step.abs()))  # softplus
    y = state_space(x.reshape(T, H, dv), B.reshape(T, G, n), C.reshape(T, G, n), step, torch.exp(W("A_log")), W("D"))
    y = rms_parts(y.reshape(T, -1) * silu(z), m["norm_groups"], eps) * W("norm")
    return y @ W("o").t()


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H] -> [T, H, dv]."""
    T, H, d = q.shape
    out = torch.empty_like(v)
    for h in range(H):
        S, n, m = q.new_zeros(d, v.shape[2]), q.new_zeros(d), q.new_zeros(())
        for t in range(T):
            new = torch.maximum(f[t, h] + m, i[t, h])
            keep, add = torch.exp(f[t, h] + m - new), torch.exp(i[t, h] - new)
            S, n, m = keep * S + add * torch.outer(k[t, h], v[t, h]), keep * n + add * k[t, h], new
            out[t, h] = (S.t() @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm(h, W, m, eps):
    T, H, d, cap = h.shape[0], m["heads"], m["dim"], m["gate_cap"]
    soft = lambda z: cap * torch.tanh(z / cap)  # noqa: E731
    i, f = soft(h @ W("i").t() + W("i.b")), log_sigmoid(soft(h @ W("f").t() + W("f.b")))
    q, k, v = ((h @ W(n).t()).view(T, H, -1) for n in "qkv")
    y = rms_parts(matrix_memory(q * d**-0.5, k, v, i, f), 1, eps).reshape(T, -1)
    return (y * W("norm") * torch.sigmoid(h @ W("g").t())) @ W("o").t()


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * rms_parts(z, 1, eps) + b * rms_parts(z**2, 1, eps) + c * rms_parts(z**3, 1, eps) + e


def dense(h, W, eps):
    return poly_norm(h @ W("up").t(), W("act"), eps) @ W("down").t()


def choose(s, top, groups):
    """Experts of one token by its scores: the best of the best groups."""
    per = s.shape[0] // groups["count"]
    value = [float(s[g * per : (g + 1) * per].sort(descending=True).values[:2].sum()) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: -value[g])[: groups["keep"]]
    allowed = [e for g in kept for e in range(g * per, (g + 1) * per)]
    return sorted(allowed, key=lambda e: -float(s[e]))[:top]


def experts(h, W, f):
    r = f["router"]
    s = torch.sigmoid(h @ W("router").t())
    out = []
    for t in range(h.shape[0]):
        y = 0
        for e in choose(s[t], r["top"], r.get("groups") or dict(count=1, keep=1)):
            y = y + s[t, e] * ((silu(h[t] @ W(f"e{e}.gate").t()) * (h[t] @ W(f"e{e}.up").t())) @ W(f"e{e}.down").t())
        out.append(y)
    return torch.stack(out)


def forward(config, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: list that receives the residual stream after every layer."""
    weight = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps, parts = config["norm"]["eps"], config["norm"]["groups"]
    norm = lambda y, name: rms_parts(y, parts, eps) * weight(name)  # noqa: E731
    x = weight("embed")[list(tokens)]
    shared = {}
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        W = lambda n: weight(f"{p}mix.{n}")  # noqa: E731, B023
        if layer["type"] == "attention":
            j = m.get("kv_from")
            shared[i] = attention_keys(x, W, m, eps) if j is None else shared[j]
            y = attention(x, W, m, eps, shared[i])
        else:
            y = {"mamba2": mamba2, "mlstm": mlstm}[layer["type"]](x, W, m, eps)
        x = x + norm(y, p + "norm1")
        if f is not None:
            F = lambda n: weight(f"{p}mlp.{n}")  # noqa: E731, B023
            x = x + norm(dense(x, F, eps) if f["kind"] == "dense" else experts(x, F, f), p + "norm2")
        if layers_out is not None:
            layers_out.append(x.clone())
    z, cap = norm(x, "final.norm") @ weight("head").t(), config.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z


def error(got, want):
    """Largest root-mean-square difference of a row, mean taken off, relative to the rows' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())

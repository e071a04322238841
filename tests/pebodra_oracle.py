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


# ------------------------------------------------------------------------------- models for the tests
def attn(heads, kv_heads, dim, vdim, window, rot, base=1e4, scale=None, diff=0.4, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), rot=dict(dims=rot, base=base),
             scale=scale or dim**-0.5, diff=diff)  # fmt: skip
    return dict(m, kv_from=kv_from) if kv_from is not None else m


def ssm(heads, groups, state, vdim, conv=4, norm_groups=1):
    return dict(heads=heads, groups=groups, state=state, vdim=vdim, conv=conv, norm_groups=norm_groups)


def memory(heads, dim, vdim, gate_cap=12.0):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap)


def plain(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, groups=(1, 1)):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=groups[0], keep=groups[1])))


def _kind(m):
    return "mamba2" if "state" in m else "mlstm" if "gate_cap" in m else "attention"


def model(width, vocab, layers, norm_groups=1, eps=1e-5, softcap=20.0):
    """``layers``: (mixer, feed-forward or None)."""
    return dict(architecture="Pebodra", width=width, vocab=vocab, norm=dict(eps=eps, groups=norm_groups), logit_softcap=softcap,
                layers=[dict(type=_kind(m), mixer=m, mlp=f) for m, f in layers])  # fmt: skip


CONFIGS = {
    # every mixer twice with different geometry, shared keys under another window, layers without a feed-forward
    "mixed": model(96, 203, [
        (ssm(6, 2, 24, 16, 4, 3), plain(112)), (attn(4, 2, 16, 24, 21, 12, 5e3, diff=0.3), moe(8, 3, 32, (4, 2))), (memory(3, 20, 28, 8.0), None),
        (attn(4, 2, 16, 24, 50, 12, 5e3, scale=0.4, diff=0.6, kv_from=1), moe(9, 2, 24, (3, 2))), (attn(6, 1, 24, 16, 33, 24), plain(56)),
        (memory(4, 8, 16), moe(4, 4, 16)), (ssm(4, 4, 16, 24, 2, 2), None), (attn(6, 1, 24, 16, 9, 24, kv_from=4), plain(40))],
        norm_groups=3, eps=3e-4, softcap=9.0),
    # equal heads, sizes of a power of two, a window of a page
    "even": model(64, 128, [(attn(4, 2, 16, 32, 16, 16), moe(8, 2, 32, (2, 1))), (ssm(4, 2, 16, 32, 4, 2), plain(128)), (memory(4, 16, 32), moe(8, 2, 32)),
                            (attn(4, 2, 16, 32, 64, 16, kv_from=0), None)], norm_groups=4),
    # widths that no 16-byte copy divides
    "odd": model(90, 77, [(attn(3, 3, 10, 13, 7, 6, 50.0), plain(37)), (ssm(3, 1, 9, 7, 3, 3), moe(6, 2, 13, (3, 1))), (memory(3, 5, 11, 4.0), plain(21)),
                          (attn(3, 3, 10, 13, 11, 6, 50.0, diff=0.7, kv_from=0), moe(5, 1, 9))], norm_groups=2, eps=1e-3, softcap=3.0),
    # one head, one expert, one tap; eps large enough to matter; no cap
    "single": model(40, 33, [(attn(1, 1, 16, 8, 5, 4, 100.0, diff=0.1), moe(1, 1, 24)), (ssm(1, 1, 16, 40, 1), None), (memory(1, 8, 4), moe(2, 1, 8, (2, 1)))],
                    eps=0.1, softcap=None),
    # no attention at all, many taps
    "states": model(48, 61, [(ssm(4, 2, 40, 12, 7, 2), plain(30)), (memory(2, 40, 72), plain(64)), (ssm(2, 2, 8, 68, 4), None)], norm_groups=6),
}  # fmt: skip


def random_tensors(name_or_config, seed=0, sharp=2.5, dtype=torch.float32):
    """Random weights under the checkpoint's names. ``sharp`` scales the query and key norms, so that single keys dominate the softmax; the
    recurrences forget slowly."""
    config = CONFIGS[name_or_config] if isinstance(name_or_config, str) else name_or_config
    g = torch.Generator().manual_seed(seed)
    D, out = config["width"], {}

    def rand(*s, gain=1.0, mean=0.0):
        return torch.randn(*s, generator=g) * gain + mean

    def mat(name, n, cols, gain=1.0):
        out[name] = rand(n, cols, gain=gain * cols**-0.5)

    out["embed"], out["final.norm"] = rand(config["vocab"], D), rand(D, gain=0.3, mean=1.0)
    mat("head", config["vocab"], D, 4.0)
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        q, H, dv = p + "mix.", m["heads"], m["vdim"]
        out[p + "norm1"] = rand(D, gain=0.3, mean=0.8)
        if layer["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            rows = dict(q=H * 2 * d) if "kv_from" in m else dict(q=H * 2 * d, k=G * 2 * d, v=G * dv)
            for n, r in rows.items():
                mat(q + n, r, D)
                out[f"{q}{n}.b"] = rand(r, gain=0.3)
                if n != "v":
                    out[f"{q}{n}.norm"] = rand(d, gain=0.3, mean=1.0) * sharp**0.5
            for n in ("lq1", "lk1", "lq2", "lk2"):
                out[q + n] = rand(d, gain=0.4 * d**-0.25)
            out[q + "o.b"] = rand(D, gain=0.3)
        elif layer["type"] == "mamba2":
            ch = H * dv + 2 * m["groups"] * m["state"]
            mat(q + "in", H * dv + ch + H, D)
            out[q + "conv"], out[q + "conv.b"] = rand(ch, m["conv"], gain=0.7 * m["conv"] ** -0.5, mean=0.1), rand(ch, gain=0.2)
            out[q + "dt_bias"], out[q + "A_log"], out[q + "D"] = rand(H, mean=-2.0), rand(H, gain=0.7, mean=-1.0), rand(H, gain=0.5, mean=0.5)
            out[q + "norm"] = rand(H * dv, gain=0.3, mean=1.0)
        else:
            for n, r in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * dv), ("g", H * dv), ("i", H), ("f", H)):
                mat(q + n, r, D)
            out[q + "i.b"], out[q + "f.b"] = rand(H, gain=0.5), rand(H, gain=1.0, mean=3.0)
            out[q + "norm"] = rand(H * dv, gain=0.3, mean=1.0)
        mat(q + "o", D, H * dv)
        if f is None:
            continue
        out[p + "norm2"] = rand(D, gain=0.3, mean=0.8)
        if f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], D)
            mat(p + "mlp.down", D, f["ff"])
            out[p + "mlp.act"] = rand(4, gain=0.3, mean=0.5)
            continue
        for e in range(f["router"]["experts"]):
            for n in ("gate", "up"):
                mat(f"{p}mlp.e{e}.{n}", f["expert"]["ff"], D)
            mat(f"{p}mlp.e{e}.down", D, f["expert"]["ff"])
        mat(p + "mlp.router", f["router"]["experts"], D, 2.0)
    return {k: v.to(dtype) for k, v in out.items()}


def random_tokens(config, n, seed=0):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

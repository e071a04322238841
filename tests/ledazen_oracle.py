"""Plain, slow definition of the Ledazen decoder, one function per mechanism, float64 by default.

No batching, no cache, no chunks: every function takes one whole sequence and writes the equation down, the recurrence
token by token. It shares no code with the product path and is what the tests of that path are compared with.
"""

from __future__ import annotations

import math

import torch


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token: a hash of it and its predecessor; the extra last row for the first token."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * mul_prev + cur * mul_cur) % buckets)
    return rows


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_around_one(x, w, eps):
    """The stored weight is the deviation from one."""
    return rms(x, eps) * (1 + w)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0)


def short_conv(x, w):
    """Per channel: y[t] = sum_s w[taps - 1 - s] x[t - s], zeros before the start; then silu."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for s in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - s] * x[t - s]
    return silu(y)


def rotate_pairs(x, dims, base):
    """x [T, heads, d] of positions 0..T-1: coordinates (2i, 2i + 1) turned by position * base^(-2i / dims), i < dims / 2."""
    out = x.clone()
    for p in range(x.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2 * i / dims)
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            out[p, :, 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[p, :, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def attention(h, W, spec, eps):
    """Grouped-query attention, q and k normed and turned; the softmax has one extra unit in its denominator."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (h @ W("q").t()).view(T, H, d), (h @ W("k").t()).view(T, G, d), (h @ W("v").t()).view(T, G, dv)
    q, k = rms(q, eps) * W("q.norm"), rms(k, eps) * W("k.norm")
    q, k = (rotate_pairs(x, spec["rot"]["dims"], spec["rot"]["base"]) for x in (q, k))
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        score = ((q[:, head] @ k[:, g].t()) * spec["scale"]).masked_fill(later, float("-inf"))
        weight = torch.softmax(torch.cat([score, torch.zeros(T, 1, dtype=h.dtype)], 1), -1)[:, :T]
        out[:, head] = weight @ v[:, g]
    return out.reshape(T, H * dv) @ W("o").t()


def delta_rule(q, k, v, decay, beta):
    """One head, token by token: q, k, decay [T, d], v [T, dv], beta [T] -> [T, dv]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.t() @ q[t])
    return torch.stack(out)


def delta(h, W, spec, eps, per_channel):
    """``per_channel`` True: a decay per key channel and a sigmoid gate, both through low-rank pairs; False: a decay per head
    and a silu gate of full rank."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (short_conv(h @ W(n).t(), W(n + ".conv")) for n in "qkv")
    q, k, v = q.view(T, G, d), k.view(T, G, d), v.view(T, H, dv)
    q, k = unit(q) * d**-0.5, unit(k)
    beta = torch.sigmoid(h @ W("b").t())
    rate = torch.exp(W("A_log"))
    if per_channel:
        z = softplus((h @ W("a1").t()) @ W("a2").t() + W("dt_bias")).view(T, H, d)
        gate = torch.sigmoid((h @ W("g1").t()) @ W("g2").t())
    else:
        z = softplus(h @ W("a").t() + W("dt_bias")).view(T, H, 1).expand(T, H, d)
        gate = silu(h @ W("g").t())
    decay = torch.exp(-rate[None, :, None] * z)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        o = delta_rule(q[:, g], k[:, g], v[:, head], decay[:, head], beta[:, head])
        out[:, head] = rms(o, eps) * W("norm")
    return (out.reshape(T, H * dv) * gate) @ W("o").t()


def mixer(h, W, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "delta":
        return delta(h, W, m, eps, False)
    assert layer["type"] == "parallel"
    left = attention(h, lambda n: W("left." + n), m["left"], eps)
    right = delta(h, lambda n: W("right." + n), m["right"], eps, True)
    return m["left_scale"] * left + m["right_scale"] * right


def feed_forward(h, w_up, w_down):
    return relu_squared(h @ w_up.t()) @ w_down.t()


def forward(config, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: list that receives the residual stream after every layer."""
    W = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps, b = config["norm"]["eps"], config["embedding"]["bigram"]
    tokens = list(tokens)
    x = W("embed")[tokens] + W("bigram")[bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = rms_around_one(x, W(p + "norm1"), eps)
        y = mixer(h, lambda n: W(f"{p}mix.{n}"), layer, eps)
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            y = y + feed_forward(h, W(p + "mlp.up"), W(p + "mlp.down"))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_around_one(x, W("final.norm"), eps) @ W("head").t()


def error(got, want):
    """Largest root-mean-square difference of a row, mean taken off, relative to the rows' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())


# ------------------------------------------------------------------------------- models for the tests
def attn(heads, kv_heads, dim, vdim, dims, base=1e4, scale=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(dims=dims, base=base), scale=scale if scale is not None else dim**-0.5)


def rule(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def both(left, right, left_scale=0.8, right_scale=0.7):
    return dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale)


def model(width, vocab, bigram, layers, eps=1e-5):
    """``bigram``: (buckets, mul_prev, mul_cur); ``layers``: (mixer, width of the feed-forward or None)."""
    return dict(architecture="Ledazen", width=width, vocab=vocab, norm=dict(eps=eps),
                embedding=dict(bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))),
                layers=[dict(type="parallel" if "left" in m else "delta", mixer=m, mlp=None if ff is None else dict(kind="dense", ff=ff))
                        for m, ff in layers])  # fmt: skip


CONFIGS = {
    # layers of different geometry and order, layers without a feed-forward, partial rotation, several groupings and taps
    "mixed": model(96, 203, (41, 13, 5), [
        (both(attn(6, 2, 32, 24, 20, scale=0.4), rule(6, 3, 24, 40, 4)), 80), (rule(4, 2, 16, 40, 3), None),
        (rule(6, 1, 40, 16, 5), 56), (both(attn(5, 5, 16, 48, 16, 5e5), rule(2, 2, 40, 8, 2), 1.3, -0.4), None)], eps=3e-4),
    # equal attention heads (one cache slab), one tap: no convolution state
    "equal": model(64, 128, (64, 3, 1), [(both(attn(4, 1, 32, 32, 32), rule(2, 1, 16, 32, 1)), 96),
                                         (both(attn(4, 1, 32, 32, 32), rule(4, 4, 32, 16, 4)), 64)]),
    # widths that no 16-byte copy divides
    "odd": model(90, 77, (23, 7, 11), [(rule(3, 3, 10, 14, 4), 50), (both(attn(6, 3, 10, 22, 6), rule(3, 1, 9, 7, 3), 0.5, 1.0), 45)], eps=1e-3),
    # one head of each kind; eps large enough to matter
    "single": model(40, 33, (9, 2, 3), [(both(attn(1, 1, 16, 48, 4, 100.0), rule(1, 1, 16, 24, 6), 1.0, 1.0), 24)], eps=0.1),
    # no attention: nothing is kept per token
    "rules": model(48, 60, (31, 5, 7), [(rule(2, 1, 24, 24, 4), 40), (rule(3, 3, 16, 32, 2), None)]),
}  # fmt: skip


def random_tensors(config, seed=0, sharp=2.5, dtype=torch.float32):
    """Random weights under the checkpoint's names. ``sharp`` scales the query and key norms, so that single keys dominate
    the softmax; decays are close to one, so that old writes are still read."""
    g = torch.Generator().manual_seed(seed)
    D, out, b = config["width"], {}, config["embedding"]["bigram"]

    def rand(*s, gain=1.0, mean=0.0):
        return torch.randn(*s, generator=g) * gain + mean

    def mat(name, rows, cols, gain=1.0):
        out[name] = rand(rows, cols, gain=gain * cols**-0.5)

    out["embed"], out["bigram"] = rand(config["vocab"], D, mean=0.3), rand(b["buckets"] + 1, D)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = rand(D, gain=0.3)
        if layer["type"] == "parallel":
            a, q = m["left"], p + "mix.left."
            mat(q + "q", a["heads"] * a["dim"], D)
            mat(q + "k", a["kv_heads"] * a["dim"], D)
            mat(q + "v", a["kv_heads"] * a["vdim"], D)
            mat(q + "o", D, a["heads"] * a["vdim"])
            for n in "qk":
                out[f"{q}{n}.norm"] = rand(a["dim"], gain=0.3, mean=1.0) * sharp**0.5
        r, q = (m["right"], p + "mix.right.") if layer["type"] == "parallel" else (m, p + "mix.")
        H, dv = r["heads"], r["vdim"]
        for n, rows in (("q", r["kv_heads"] * r["dim"]), ("k", r["kv_heads"] * r["dim"]), ("v", H * dv)):
            mat(q + n, rows, D)
            out[f"{q}{n}.conv"] = rand(rows, r["conv"], gain=0.6)
        mat(q + "b", H, D)
        out[q + "A_log"], out[q + "norm"] = rand(H, gain=0.5), rand(dv, gain=0.3, mean=1.0)
        if layer["type"] == "parallel":
            for n, rows, rank in (("a", H * r["dim"], 5 + i), ("g", H * dv, 11 - i)):  # inner widths are a matter of the tensors
                mat(f"{q}{n}1", rank, D)
                mat(f"{q}{n}2", rows, rank)
            out[q + "dt_bias"] = rand(H * r["dim"], mean=-3.5)
        else:
            mat(q + "a", H, D)
            mat(q + "g", H * dv, D)
            out[q + "dt_bias"] = rand(H, mean=-3.5)
        mat(q + "o", D, H * dv)
        if layer["mlp"] is not None:
            mat(p + "mlp.up", layer["mlp"]["ff"], D)
            mat(p + "mlp.down", D, layer["mlp"]["ff"], 0.7)
    out["final.norm"] = rand(D, gain=0.3)
    mat("head", config["vocab"], D)
    return {k: v.to(dtype) for k, v in out.items()}


def shapes(tensors):
    return {k: tuple(v.shape) for k, v in tensors.items()}


def random_tokens(config, n, seed=0):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

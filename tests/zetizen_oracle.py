"""Plain, slow definition of the Zetizen decoder, one function per mechanism, float64 by default.

No batching, no cache: every function takes one whole sequence and writes the equation down. It shares no code with the
product path and is what the tests of that path are compared with.
"""

from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def bucket(n, rows, far):
    """Row of the distance table for distance ``n``: one row each up to half the rows, then rows that grow geometrically up to
    distance ``far``, the last row beyond."""
    half = rows // 2
    if n < half:
        return n
    x = math.log(n / half) / math.log(far / half) * (rows - half)
    near = round(x)
    step = near if abs(x - near) < 1e-9 else math.floor(x)  # a distance on an edge belongs to the bucket that starts there
    return min(rows - 1, half + step)


def distance_bias(table, T, far):
    """[heads, T, T]: what head h adds to the score of query i and key j <= i."""
    rows = torch.tensor([bucket(n, table.shape[0], far) for n in range(T)])
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return table[rows[(i - j).clamp(min=0)]].permute(2, 0, 1)


def causal(T):
    return torch.ones(T, T, dtype=torch.bool).tril()


def chunk_mask(T, size):
    c = torch.arange(T) // size
    return causal(T) & (c[:, None] == c[None, :])


def yarn(dims, base, scaling):
    """Frequencies of the dims / 2 pairs and the factor of their cosines and sines; ``scaling`` None: no stretching."""
    freq = [base ** (-2 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0
    turn = lambda t: dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0), 1)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate_halves(x, rot):
    """x [T, heads, d] of positions 0..T-1: coordinates (i, i + dims / 2) turned by position * frequency i."""
    half, out = rot["dims"] // 2, x.clone()
    freq, gain = yarn(rot["dims"], rot["base"], rot.get("scaling"))
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * torch.tensor(freq, dtype=torch.float64)
    c, s = angle.cos() * gain, angle.sin() * gain
    u, v = x[..., :half], x[..., half : 2 * half]
    out[..., :half], out[..., half : 2 * half] = u * c - v * s, v * c + u * s
    return out


def attend(q, k, v, scale, see, cap=None, bias=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], see [T, T] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        if cap is not None:
            s = soft_cap(s, cap)
        if bias is not None:
            s = s + bias[h]
        out.append(torch.softmax(s.masked_fill(~see, float("-inf")), -1) @ v[:, g])
    return torch.stack(out, 1)


def biased_attention(h, W, m, eps):
    """No positions but a learned bias by distance."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = rms(h @ W("q").t(), W("q.norm"), eps), rms(h @ W("k").t(), W("k.norm"), eps), h @ W("v").t()
    q, k, v = q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1)
    y = attend(q, k, v, m["scale"], causal(T), m["softcap"], distance_bias(W("rel"), T, m["bias_max"]))
    return y.reshape(T, -1) @ W("o").t()


def chunked_attention(h, W, m, eps):
    """Keys and values are one projection; queries see the keys of their own chunk."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = h @ W("q").t() + W("q.b"), h @ W("k").t() + W("k.b")
    v = k.view(T, G, -1)
    q, k = rms(q, W("q.norm"), eps).view(T, H, -1), rms(k, W("k.norm"), eps).view(T, G, -1)
    y = attend(rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"]), v, m["scale"], chunk_mask(T, m["mask"]["size"]), m["softcap"])
    y = y * torch.sigmoid(h @ W("g").t())[:, :, None]
    return y.reshape(T, -1) @ W("o").t()


def latent_attention(h, W, m, eps):
    T, H, d, r, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (rms(h @ W("dq").t(), W("dq.norm"), eps) @ W("uq").t()).view(T, H, d + r)
    down = h @ W("dkv").t()
    c = rms(down[:, :R], W("dkv.norm"), eps)
    turned = rotate_halves(down[:, None, R:], m["rot"]).expand(T, H, r)
    k = torch.cat([(c @ W("uk").t()).view(T, H, d), turned], -1)
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], m["rot"])], -1)
    y = attend(q, k, (c @ W("uv").t()).view(T, H, -1), m["scale"], causal(T))
    return (y.reshape(T, -1) * torch.sigmoid(h @ W("g").t())) @ W("o").t()


MIXERS = {"attention": biased_attention, "attention_2": chunked_attention, "latent_attention": latent_attention}


def feed_forward(h, gate, up, down):
    return (silu(h @ gate.t()) * (h @ up.t())) @ down.t()


def experts(h, W, f):
    """Router with a bias, softmax over the chosen logits; an expert for every token beside them."""
    z = h @ W("router").t() + W("router.b")
    top, which = torch.topk(z, f["router"]["top"], dim=-1)
    weight, ff = torch.softmax(top, -1), lambda e, x: feed_forward(x, W(e + ".gate"), W(e + ".up"), W(e + ".down"))
    out = []
    for t in range(h.shape[0]):
        out.append(sum(weight[t, j] * ff(f"e{int(which[t, j])}", h[t]) for j in range(top.shape[1])))
    y = torch.stack(out)
    return y + ff("shared", h) if f.get("shared") else y


def forward(config, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: list that receives the residual stream after every layer."""
    W = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    x = layer_norm(W("embed")[list(tokens)], W("embed.norm"), eps)
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = layer_norm(x, W(p + "norm1"), eps)
        y = MIXERS[layer["type"]](h, lambda n: W(f"{p}mix.{n}"), layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + experts(h, lambda n: W(f"{p}mlp.{n}"), layer["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W("final.norm"), eps) @ W("embed").t() * config["logit_scale"]


def error(got, want):
    """Largest root-mean-square difference of a row, mean taken off, relative to the rows' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())


# ------------------------------------------------------------------------------- models for the tests
def yarn_rot(dims, base=1e4, factor=4.0, original=64, fast=8.0, slow=1.0):
    return dict(dims=dims, base=base, scaling=dict(factor=factor, original=original, fast=fast, slow=slow))


def biased(heads, kv_heads, dim, vdim, rows, far, scale=None, cap=9.0):
    """``rows``: distance buckets (a matter of the tensor, not of the configuration)."""
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, bias_max=far, scale=scale or dim**-0.5, softcap=cap, _rows=rows)


def chunked(heads, kv_heads, dim, size, rot, scale=None, cap=12.0):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=size), rot=rot, scale=scale or dim**-0.5, softcap=cap)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, rot=None, scale=None):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=rot or yarn_rot(rot_dim),
                scale=scale or (dim + rot_dim) ** -0.5)  # fmt: skip


def moe(experts, top, ff, shared=0):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top), **({"shared": dict(ff=shared)} if shared else {}))


def _kind(m):
    return "latent_attention" if "kv_rank" in m else "attention" if "bias_max" in m else "attention_2"


def model(width, vocab, layers, eps=1e-5, logit_scale=1.5):
    """``layers``: (mixer, feed-forward or None). Returns (config, distance buckets by layer)."""
    plain = lambda m: {k: v for k, v in m.items() if k != "_rows"}  # noqa: E731
    config = dict(architecture="Zetizen", width=width, vocab=vocab, norm=dict(eps=eps), logit_scale=logit_scale,
                  layers=[dict(type=_kind(m), mixer=plain(m), mlp=f) for m, f in layers])  # fmt: skip
    return config, {i: m["_rows"] for i, (m, _) in enumerate(layers) if "_rows" in m}


MODELS = {
    # every mixer twice with different geometry and order, layers without a feed-forward, one without a shared expert
    "mixed": model(96, 203, [
        (latent(3, 24, 16, 40, 32, 48), moe(6, 2, 32, 56)), (chunked(6, 2, 32, 20, yarn_rot(20, 5e3), cap=5.0), None),
        (biased(6, 3, 24, 40, 10, 33), moe(5, 3, 48)), (biased(4, 4, 16, 24, 24, 100, cap=30.0), moe(4, 4, 16, 24)),
        (latent(5, 16, 8, 24, 40, 24, yarn_rot(8, 100.0, 2.0, 32, 4.0, 0.5)), None), (chunked(4, 1, 16, 33, yarn_rot(16)), moe(7, 1, 24, 40))],
        eps=3e-4, logit_scale=0.7),
    # equal heads, sizes of a power of two; chunks of a page
    "even": model(64, 128, [(biased(4, 2, 32, 32, 16, 64), moe(8, 2, 32, 64)), (chunked(4, 2, 32, 16, yarn_rot(32)), moe(8, 2, 32, 64)),
                            (latent(4, 32, 16, 32, 48, 64), moe(8, 2, 32, 64))]),
    # widths that no 16-byte copy divides
    "odd": model(90, 77, [(biased(3, 3, 10, 14, 6, 17), moe(5, 2, 21, 13)), (latent(3, 10, 6, 7, 11, 19), moe(3, 2, 9, 5)),
                          (chunked(6, 3, 10, 7, yarn_rot(6, 50.0)), moe(5, 2, 17, 11))], eps=1e-3, logit_scale=3.0),
    # one head, one expert; eps large enough to matter
    "single": model(40, 33, [(biased(1, 1, 16, 48, 2, 5), moe(1, 1, 24, 16)), (chunked(1, 1, 16, 5, yarn_rot(4, 100.0)), None),
                             (latent(1, 16, 4, 24, 8, 16), moe(2, 1, 8))], eps=0.1, logit_scale=1.0),
}  # fmt: skip


def random_tensors(name_or_model, seed=0, sharp=2.5, dtype=torch.float32):
    """Random weights under the checkpoint's names. ``sharp`` scales the query and key norms, so that single keys dominate the
    softmax."""
    config, rows = MODELS[name_or_model] if isinstance(name_or_model, str) else name_or_model
    g = torch.Generator().manual_seed(seed)
    D, out = config["width"], {}

    def rand(*s, gain=1.0, mean=0.0):
        return torch.randn(*s, generator=g) * gain + mean

    def mat(name, n, cols, gain=1.0):
        out[name] = rand(n, cols, gain=gain * cols**-0.5)

    out["embed"], out["embed.norm"], out["final.norm"] = rand(config["vocab"], D, mean=0.3), rand(D, gain=0.3, mean=1.0), rand(D, gain=0.3, mean=0.2)
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        q = p + "mix."
        out[p + "norm1"] = rand(D, gain=0.3, mean=1.0)
        H, dv = m["heads"], m["vdim"]
        if layer["type"] == "latent_attention":
            mat(q + "dq", m["q_rank"], D)
            mat(q + "dkv", m["kv_rank"] + m["rot_dim"], D)
            out[q + "dq.norm"], out[q + "dkv.norm"] = rand(m["q_rank"], gain=0.3, mean=sharp), rand(m["kv_rank"], gain=0.3, mean=1.0)
            mat(q + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            mat(q + "uk", H * m["dim"], m["kv_rank"])
            mat(q + "uv", H * dv, m["kv_rank"])
            mat(q + "g", H * dv, D)
        else:
            G, d = m["kv_heads"], m["dim"]
            mat(q + "q", H * d, D)
            mat(q + "k", G * d, D)
            for n, w in (("q", H * d), ("k", G * d)):
                out[f"{q}{n}.norm"] = rand(w, gain=0.3, mean=1.0) * sharp**0.5
            if layer["type"] == "attention":
                mat(q + "v", G * dv, D)
                out[q + "rel"] = rand(rows[i], H, gain=1.5)
            else:
                out[q + "q.b"], out[q + "k.b"] = rand(H * d, gain=0.5), rand(G * d, gain=0.5)
                mat(q + "g", H, D)
        mat(q + "o", D, H * dv)
        if f is not None:
            stems = [(f"{p}mlp.e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
            stems += [(p + "mlp.shared", f["shared"]["ff"])] if f.get("shared") else []
            for s, ff in stems:
                mat(s + ".gate", ff, D)
                mat(s + ".up", ff, D)
                mat(s + ".down", D, ff)
            mat(p + "mlp.router", f["router"]["experts"], D, 2.0)
            out[p + "mlp.router.b"] = rand(f["router"]["experts"], gain=0.7)
    return {k: v.to(dtype) for k, v in out.items()}


def shapes(tensors):
    return {k: tuple(v.shape) for k, v in tensors.items()}


def random_tokens(config, n, seed=0):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

"""Plain, slow definition of the Pefolix decoder, one function per mechanism, float64 by default.

No batching, no cache, no chunks: every function takes one whole sequence and writes the equation down. It shares no
code with the product path and is what the tests of that path are compared with.
"""

from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    """Weight-only layer norm over the last axis; the variance is the mean of the squared deviations."""
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z**3)))


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def distance_slopes(heads):
    """Per-head factor of the linear distance penalty: 2^(-8/H), 2^(-16/H), ..., 2^-8."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def visible(i, j, size, keep_first):
    """Causal sliding window of ``size`` tokens (the own token included) plus the first ``keep_first`` tokens."""
    return j <= i and (i - j < size or j < keep_first)


def attention(h, w_q, w_k, w_v, w_o, spec):
    """Grouped-query attention with a windowed mask and a linear distance penalty, written position by position."""
    T, H, G, d, dv = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (h @ w_q.t()).view(T, H, d), (h @ w_k.t()).view(T, G, d), (h @ w_v.t()).view(T, G, dv)
    slopes = distance_slopes(H)
    pos = torch.arange(T)
    dist = pos[:, None] - pos[None, :]
    see = (dist >= 0) & ((dist < spec["mask"]["size"]) | (pos[None, :] < spec["mask"]["keep_first"]))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        score = (q[:, head] @ k[:, g].t()) * spec["scale"] - slopes[head] * dist.to(h.dtype)
        weight = torch.softmax(score.masked_fill(~see, float("-inf")), dim=-1)
        out[:, head] = weight @ v[:, g]
    return out.reshape(T, H * dv) @ w_o.t()


def dense_ff(h, w_gate, w_up, w_down):
    return (gelu_tanh(h @ w_gate.t()) * (h @ w_up.t())) @ w_down.t()


def small_ff(h, w_up, w_down):
    """An expert: no gate, squared relu."""
    return relu_squared(h @ w_up.t()) @ w_down.t()


def route(h, w_router, top):
    """Softmax over all experts; the largest ``top`` are used with their own scores as weights."""
    score = torch.softmax(h @ w_router.t(), dim=-1)
    weight, index = torch.topk(score, top, dim=-1)
    return weight, index


def mixture(h, w_router, experts, top, shared=None, w_sg=None):
    """``experts``: list of (up, down). ``shared``: (up, down) of the always-on expert, scaled by sigmoid(w_sg h)."""
    weight, index = route(h, w_router, top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(top):
            up, down = experts[int(index[t, j])]
            out[t] += weight[t, j] * small_ff(h[t], up, down)
    if shared is not None:
        out = out + torch.sigmoid(h @ w_sg.t()) * small_ff(h, *shared)
    return out


def forward(config, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: list that receives the residual stream after every layer."""
    W = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    x = W("embed")[torch.as_tensor(tokens)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        assert layer["type"] == "attention"
        y = attention(layer_norm(x, W(p + "norm1"), eps), W(p + "mix.q"), W(p + "mix.k"), W(p + "mix.v"), W(p + "mix.o"), layer["mixer"])
        x = x + layer_norm(y, W(p + "norm1b"), eps)
        mlp = layer["mlp"]
        if mlp is not None:
            h = layer_norm(x, W(p + "norm2"), eps)
            if mlp["kind"] == "dense":
                y = dense_ff(h, W(p + "mlp.gate"), W(p + "mlp.up"), W(p + "mlp.down"))
            else:
                experts = [(W(f"{p}mlp.e{e}.up"), W(f"{p}mlp.e{e}.down")) for e in range(mlp["router"]["experts"])]
                shared = (W(p + "mlp.shared.up"), W(p + "mlp.shared.down")) if mlp.get("shared") else None
                y = mixture(h, W(p + "mlp.router"), experts, mlp["router"]["top"], shared, W(p + "mlp.shared.sg") if shared else None)
            x = x + layer_norm(y, W(p + "norm2b"), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W("final.norm"), eps) @ W("head").t()


# ------------------------------------------------------------------------------- models for the tests
def attn(heads, kv_heads, dim, vdim, size, keep, scale=None):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else dim**-0.5,
                mask=dict(size=size, keep_first=keep))  # fmt: skip


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, shared=None):
    d = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    return dict(d, shared=dict(ff=shared)) if shared else d


def model(width, vocab, layers, eps=1e-5):
    return dict(architecture="Pefolix", width=width, vocab=vocab, norm=dict(eps=eps),
                layers=[dict(type="attention", mixer=a, mlp=m) for a, m in layers])  # fmt: skip


CONFIGS = {
    # layers of different geometry, a mixer-only layer, several groupings, key and value heads of different width
    "mixed": model(96, 203, [(attn(6, 2, 32, 24, 21, 4), dense(80)), (attn(4, 4, 16, 40, 9, 0), None),
                             (attn(8, 1, 24, 16, 33, 2, scale=0.31), moe(40, 7, 2, shared=24)), (attn(2, 1, 64, 8, 1, 3), moe(16, 5, 1)),
                             (attn(5, 5, 8, 72, 40, 20), dense(136))], eps=3e-4),
    # equal layers (one cache slab), every token sees a single expert of two, the window reaches past the kept tokens
    "equal": model(64, 128, [(attn(4, 2, 32, 32, 12, 5), moe(32, 2, 1, shared=48)), (attn(4, 2, 32, 32, 12, 5), dense(96)),
                             (attn(4, 2, 32, 32, 12, 5), moe(32, 2, 2))]),
    # widths that no 16-byte copy divides
    "odd": model(90, 77, [(attn(3, 3, 10, 14, 17, 1), dense(50)), (attn(6, 3, 12, 22, 25, 6), moe(18, 6, 4, shared=30))], eps=1e-3),
    # one head of each kind; eps large enough to matter
    "single": model(40, 33, [(attn(1, 1, 16, 16, 5, 1), dense(24)), (attn(1, 1, 16, 48, 300, 0), moe(8, 4, 3, shared=8))], eps=0.1),
}  # fmt: skip


def random_tensors(config, seed=0, sharp=3.0, dtype=torch.float32):
    """Random weights under the checkpoint's names. ``sharp`` scales queries and keys, so that single keys dominate the
    softmax and a key too many or too few shows."""
    g = torch.Generator().manual_seed(seed)
    D, out = config["width"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = torch.randn(rows, cols, generator=g) * gain * cols**-0.5

    def norm(name):
        out[name] = 1 + 0.3 * torch.randn(D, generator=g)

    out["embed"] = torch.randn(config["vocab"], D, generator=g) + 0.5
    for i, layer in enumerate(config["layers"]):
        p, a, m = f"l{i}.", layer["mixer"], layer["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if m is not None else ()):
            norm(p + n)
        mat(p + "mix.q", a["heads"] * a["dim"], D, sharp)
        mat(p + "mix.k", a["kv_heads"] * a["dim"], D, sharp)
        mat(p + "mix.v", a["kv_heads"] * a["vdim"], D)
        mat(p + "mix.o", D, a["heads"] * a["vdim"])
        if m is None:
            continue
        if m["kind"] == "dense":
            for n in ("gate", "up"):
                mat(f"{p}mlp.{n}", m["ff"], D)
            mat(p + "mlp.down", D, m["ff"])
            continue
        for e in [f"e{j}" for j in range(m["router"]["experts"])] + (["shared"] if m.get("shared") else []):
            ff = m["shared"]["ff"] if e == "shared" else m["expert"]["ff"]
            mat(f"{p}mlp.{e}.up", ff, D)
            mat(f"{p}mlp.{e}.down", D, ff)
        mat(p + "mlp.router", m["router"]["experts"], D, 2.0)
        if m.get("shared"):
            mat(p + "mlp.shared.sg", 1, D)
    norm("final.norm")
    mat("head", config["vocab"], D)
    return {k: v.to(dtype) for k, v in out.items()}


def random_tokens(config, n, seed=0):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Largest root-mean-square difference of a row, mean taken off, relative to the rows' spread."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())

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

"""Per-layer description of decoders whose layers differ from one another.

``ModelConfig`` describes a stack of equal layers by flat fields. A design that gives every layer its own head counts,
widths, window or feed-forward carries a list of ``LayerSpec`` instead (``ModelConfig.layer_specs``); the flat fields then
hold the largest value of each size, for code that only budgets memory. The specs are mechanism parameters, not a model:
any architecture whose layers are built from these pieces can use them.
"""

from __future__ import annotations

import dataclasses
from dataclasses import dataclass


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention without rotation. ``window``: a query at position i sees keys j with i - j < window (None:
    all earlier ones) and, whatever the distance, the first ``keep_first`` tokens of the sequence. ``distance_bias``
    "geometric": head h of H subtracts ``2^(-8 (h + 1) / H) * (i - j)`` from its scores."""

    heads: int
    kv_heads: int
    dim: int  # width of a query / key head
    vdim: int  # width of a value head
    scale: float
    window: int | None = None
    keep_first: int = 0
    distance_bias: str | None = None

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide over {self.kv_heads} key/value heads")
        if self.window is not None and self.window < 1:
            raise ValueError(f"attention window of {self.window} tokens: a query must at least see itself")
        if self.distance_bias not in (None, "geometric"):
            raise ValueError(f"unknown distance bias {self.distance_bias!r}")

    def slopes(self) -> list[float] | None:
        """Distance-penalty factor of every query head (None: no penalty)."""
        if self.distance_bias is None:
            return None
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclass(frozen=True)
class FeedForwardSpec:
    """Dense (``experts`` None) or mixture-of-experts feed-forward. ``gated``: ``down(act(gate x) * up x)``, otherwise
    ``down(act(up x))``; with experts the same form is every expert's. ``score`` / ``renorm``: router scores over all
    experts, kept as they are or divided by the sum of the chosen ones. ``shared_ff`` > 0: an expert of that width runs
    for every token, scaled by a sigmoid gate of its own when ``shared_gate``."""

    ff: int
    act: str
    gated: bool = True
    experts: int | None = None
    top: int = 1
    score: str = "softmax"
    renorm: bool = False
    shared_ff: int = 0
    shared_gate: bool = False

    def __post_init__(self):
        if self.act not in ("silu", "gelu_tanh", "relu2"):
            raise ValueError(f"unknown activation {self.act!r}")
        if self.experts is not None and not 1 <= self.top <= self.experts:
            raise ValueError(f"{self.top} of {self.experts} experts per token")

    def params(self, width: int) -> int:
        mats = 3 if self.gated else 2
        if self.experts is None:
            return mats * width * self.ff
        n = self.experts * (mats * width * self.ff + width)
        if self.shared_ff:
            n += mats * width * self.shared_ff + (width if self.shared_gate else 0)
        return n


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: FeedForwardSpec | None = None  # None: the layer is its mixer only

    @classmethod
    def of(cls, x) -> "LayerSpec":
        """Accepts a ``LayerSpec`` or its ``dataclasses.asdict`` form (presets, argument namespaces read from JSON)."""
        if isinstance(x, cls):
            return x
        mixer, mlp = x["mixer"], x.get("mlp")
        return cls(mixer if isinstance(mixer, AttentionSpec) else AttentionSpec(**mixer),
                   mlp if mlp is None or isinstance(mlp, FeedForwardSpec) else FeedForwardSpec(**mlp))  # fmt: skip

    def to_dict(self) -> dict:
        return dataclasses.asdict(self)


def flat_sizes(specs: list[LayerSpec]) -> dict:
    """The ``ModelConfig`` size fields of a specified stack: the largest value of each over the layers."""
    at, ff = [s.mixer for s in specs], [s.mlp for s in specs if s.mlp is not None]
    moe = [m for m in ff if m.experts is not None]
    out = dict(num_layers=len(specs), num_attention_heads=max(a.heads for a in at), num_query_groups=max(a.kv_heads for a in at),
               kv_channels=max(a.dim for a in at), v_head_dim=max(a.vdim for a in at),
               ffn_hidden_size=max((m.ff for m in ff if m.experts is None), default=max((m.ff for m in ff), default=1)))  # fmt: skip
    if moe:
        out.update(num_experts=max(m.experts for m in moe), moe_ffn_hidden_size=max(m.ff for m in moe),
                   moe_router_topk=max(m.top for m in moe), norm_topk_prob=False, moe_router_pre_softmax=True,
                   moe_shared_expert_intermediate_size=max(m.shared_ff for m in moe) or None)  # fmt: skip
    return out


# ------------------------------------------------------------------------------------------------- Pefolix
# Fixed by the design: layer norms before and after every sub-layer, tanh-gelu gated dense feed-forward, ungated
# squared-relu experts weighted by their own softmax score, geometric distance bias. Everything else is in config.json.


def pefolix_config(c: dict) -> dict:
    """``config.json`` of a Pefolix model -> ``ModelConfig`` arguments."""
    specs = []
    for i, layer in enumerate(c["layers"]):
        if layer["type"] != "attention":
            raise ValueError(f"layer {i}: a Pefolix model has no mixer of type {layer['type']!r}")
        m, mask, f = layer["mixer"], layer["mixer"].get("mask") or {}, layer.get("mlp")
        mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), mask.get("size"),
                              mask.get("keep_first", 0), "geometric")  # fmt: skip
        mlp = None
        if f is not None and f["kind"] == "dense":
            mlp = FeedForwardSpec(f["ff"], "gelu_tanh")
        elif f is not None and f["kind"] == "moe":
            shared = f.get("shared")
            mlp = FeedForwardSpec(f["expert"]["ff"], "relu2", gated=False, experts=f["router"]["experts"], top=f["router"]["top"],
                                  shared_ff=shared["ff"] if shared else 0, shared_gate=bool(shared))  # fmt: skip
        elif f is not None:
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        specs.append(LayerSpec(mixer, mlp))
    return dict(flat_sizes(specs), layer_specs=specs, hidden_size=c["width"], vocab_size=c["vocab"], norm_epsilon=c["norm"]["eps"],
                norm_kind="layer", post_self_attn_layernorm=True, post_mlp_layernorm=True, tie_word_embeddings=False,
                model_arch="Pefolix")  # fmt: skip


def pefolix_json(cfg) -> dict:
    """The ``config.json`` of a Pefolix ``ModelConfig`` (inverse of ``pefolix_config``)."""
    layers = []
    for s in cfg.layer_specs:
        a, m = s.mixer, s.mlp
        mixer = dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale,
                     mask=dict(size=a.window, keep_first=a.keep_first))  # fmt: skip
        mlp = None
        if m is not None and m.experts is None:
            mlp = dict(kind="dense", ff=m.ff)
        elif m is not None:
            mlp = dict(kind="moe", expert=dict(ff=m.ff), router=dict(experts=m.experts, top=m.top))
            if m.shared_ff:
                mlp["shared"] = dict(ff=m.shared_ff)
        layers.append(dict(type="attention", mixer=mixer, mlp=mlp))
    return dict(architecture="Pefolix", layers=layers, norm=dict(eps=cfg.norm_epsilon), vocab=cfg.vocab_size, width=cfg.hidden_size)


# ``config.json`` files that name their design in "architecture": name -> (reader, writer)
LAYERED_ARCHITECTURES = {"Pefolix": (pefolix_config, pefolix_json)}

"""Per-layer description of decoders whose layers differ from one another.

``ModelConfig`` describes a stack of equal layers by flat fields. A design that gives every layer its own head counts,
widths, window or feed-forward carries a list of ``LayerSpec`` instead (``ModelConfig.layer_specs``); the flat fields then
hold the largest value of each size, for code that only budgets memory. The specs are mechanism parameters, not a model:
any architecture whose layers are built from these pieces can use them.

A layer is a mixer (``AttentionSpec``, ``LatentSpec``, ``DeltaSpec``, ``StateSpaceSpec``, ``MatrixMemorySpec``, or two of them side by side:
``ParallelSpec``) and a feed-forward, one after the other with a residual sum each, or both reading one normed input
(``LayerSpec.parallel_ff``).
"""

from __future__ import annotations

import dataclasses
import math
from dataclasses import dataclass


@dataclass(frozen=True)
class YarnSpec:
    """Stretching of a rotation to ``factor`` times the ``original`` context: frequencies that turn more than ``fast`` times in it
    stay, those that turn less than ``slow`` times are divided by ``factor``, a linear ramp over the pair numbers between."""

    factor: float
    original: int
    fast: float
    slow: float

    def gain(self) -> float:
        """Factor of every cosine and sine."""
        return 0.1 * math.log(self.factor) + 1.0

    def stretched(self, dims: int, base: float) -> list[float]:
        """Share (0 to 1) of each pair's frequency that is divided by ``factor``."""
        pair = lambda turns: dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(base))  # noqa: E731
        lo, hi = max(math.floor(pair(self.fast)), 0), min(math.ceil(pair(self.slow)), dims - 1)
        return [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` coordinates of a query / key head by ``position * base^(-2i / dims)`` for pair i;
    ``interleaved``: pair i is (2i, 2i + 1), otherwise (i, i + dims / 2). ``scaling``: the frequencies are stretched."""

    dims: int
    base: float
    interleaved: bool = True
    scaling: YarnSpec | None = None

    def __post_init__(self):
        if isinstance(self.scaling, dict):
            object.__setattr__(self, "scaling", YarnSpec(**self.scaling))
        if self.dims < 0 or self.dims % 2:
            raise ValueError(f"a rotation of {self.dims} coordinates: they come in pairs")

    def frequencies(self) -> list[float]:
        """Angle per position of every pair."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.scaling is None:
            return f
        return [x / self.scaling.factor * r + x * (1.0 - r) for x, r in zip(f, self.scaling.stretched(self.dims, self.base))]

    def gain(self) -> float:
        return 1.0 if self.scaling is None else self.scaling.gain()


@dataclass(frozen=True)
class DistanceBiasSpec:
    """Learned number per (distance bucket, query head) that is added to a score: ``rows`` buckets, the first half one distance
    each, the others growing geometrically up to distance ``far``; the last one takes everything beyond."""

    rows: int
    far: int

    def __post_init__(self):
        if self.rows < 2 or self.far <= self.rows // 2:
            raise ValueError(f"{self.rows} distance buckets up to distance {self.far}: the last must lie beyond half their number")

    def bucket(self, n: int) -> int:
        half = self.rows // 2
        if n < half:
            return n
        x = math.log(n / half) / math.log(self.far / half) * (self.rows - half)
        # a distance that is exactly a bucket's first one must not fall below it by the logarithm's rounding
        return min(self.rows - 1, half + (round(x) if abs(x - round(x)) < 1e-9 else math.floor(x)))

    def by_distance(self) -> list[int]:
        """Bucket of the distances 0, 1, ...; from the last entry on it is the last bucket."""
        out = [0]
        while out[-1] < self.rows - 1:
            out.append(self.bucket(len(out)))
        return out


GATES = (None, "head", "channel")  # sigmoid gate of a mixer's output: one number per head, or one per output channel


def _gate_rows(gate: str | None, heads: int, vdim: int) -> int:
    return 0 if gate is None else heads * (vdim if gate == "channel" else 1)


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention. ``window``: a query at position i sees keys j with i - j < window (None:
    all earlier ones) and, whatever the distance, the first ``keep_first`` tokens of the sequence; ``chunk``: only keys of its
    own block of that many positions. ``softcap``: scores pass ``c tanh(score / c)``. ``distance_bias``
    "geometric": head h of H subtracts ``2^(-8 (h + 1) / H) * (i - j)`` from its scores; a ``DistanceBiasSpec``: a learned number
    is added. ``qk_norm``: RMS norm of every query and key head (one weight each, shared by the heads) before the rotation
    ``rot``; with ``norm_over`` "projection" of all heads at once, a weight per channel. ``qk_bias``: the query and key
    projections have biases, ``vo_bias``: the value and output projections have. ``tied_values``: the values are the keys as projected,
    before norm and rotation. ``gate``: see ``GATES``. ``sink``: score of an extra column of the softmax that has no value (None: no
    such column).

    ``diff``: every head is the difference of two attentions over the same values, ``o = a1 - w a2`` with a learned w per layer that
    starts out near ``diff``, over its root mean square and times ``1 - diff``; ``dim`` is then the width of each of the two query /
    key halves of a head. ``kv_from``: the keys and values are those that layer ``kv_from`` left in the cache."""

    heads: int
    kv_heads: int
    dim: int  # width of a query / key head
    vdim: int  # width of a value head
    scale: float
    window: int | None = None
    keep_first: int = 0
    distance_bias: str | DistanceBiasSpec | None = None
    qk_norm: bool = False
    rot: RotarySpec | None = None
    sink: float | None = None
    chunk: int | None = None
    softcap: float | None = None
    norm_over: str = "head"
    qk_bias: bool = False
    tied_values: bool = False
    gate: str | None = None
    vo_bias: bool = False
    diff: float | None = None
    kv_from: int | None = None

    def __post_init__(self):
        if isinstance(self.rot, dict):
            object.__setattr__(self, "rot", RotarySpec(**self.rot))
        if isinstance(self.distance_bias, dict):
            object.__setattr__(self, "distance_bias", DistanceBiasSpec(**self.distance_bias))
        if self.rot is not None and self.rot.dims > self.dim:
            raise ValueError(f"a rotation of {self.rot.dims} coordinates in a head of {self.dim}")
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide over {self.kv_heads} key/value heads")
        if self.window is not None and self.window < 1:
            raise ValueError(f"attention window of {self.window} tokens: a query must at least see itself")
        if self.chunk is not None and self.chunk < 1:
            raise ValueError(f"attention chunks of {self.chunk} tokens")
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"scores capped at {self.softcap}")
        if self.distance_bias not in (None, "geometric") and self.learned_bias is None:
            raise ValueError(f"unknown distance bias {self.distance_bias!r}")
        if self.distance_bias == "geometric" and self.softcap is not None:
            raise ValueError("a distance penalty and capped scores in one mixer")
        if self.norm_over not in ("head", "projection") or self.gate not in GATES:
            raise ValueError(f"unknown norm {self.norm_over!r} or gate {self.gate!r}")
        if self.tied_values and self.vdim != self.dim:
            raise ValueError(f"keys of width {self.dim} cannot be the values of width {self.vdim}")
        if self.diff is not None and (self.distance_bias is not None or self.sink is not None or self.gate is not None or self.tied_values
                                      or (self.qk_norm and self.norm_over != "head")):  # fmt: skip
            raise ValueError("a difference of two attentions has no distance bias, sink, gate, tied values or norm over all heads")
        if self.kv_from is not None and (self.tied_values or self.kv_from < 0):
            raise ValueError("keys and values of another layer cannot be tied")

    @property
    def learned_bias(self) -> DistanceBiasSpec | None:
        return self.distance_bias if isinstance(self.distance_bias, DistanceBiasSpec) else None

    @property
    def gate_rows(self) -> int:
        return _gate_rows(self.gate, self.heads, self.vdim)

    def cache_geometry(self, tp: int = 1) -> tuple[int, int, int]:
        """(heads, key width, value width) of what one token leaves in the cache."""
        return self.kv_heads // tp, self.maps * self.dim, self.vdim

    @property
    def maps(self) -> int:
        """Attentions per head."""
        return 1 if self.diff is None else 2

    def norm_widths(self) -> tuple[int, int]:
        """Weights of the query norm and of the key norm."""
        return (self.dim, self.dim) if self.norm_over == "head" else (self.heads * self.dim, self.kv_heads * self.dim)

    def slopes(self) -> list[float] | None:
        """Distance-penalty factor of every query head (None: no penalty)."""
        if self.distance_bias != "geometric":
            return None
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]

    def params(self, width: int) -> int:
        own, dim = (0 if self.kv_from is not None else self.kv_heads), self.maps * self.dim
        values = 0 if self.tied_values else own * self.vdim
        n = width * (self.heads * (dim + self.vdim) + own * dim + values + self.gate_rows)
        n += sum(self.norm_widths()[: 2 if own else 1]) if self.qk_norm else 0
        n += (self.heads + own) * dim if self.qk_bias else 0
        n += values + width if self.vo_bias else 0
        n += 4 * self.dim if self.diff is not None else 0
        return n + (self.learned_bias.rows * self.heads if self.learned_bias else 0)


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention: queries come from a normed latent of width ``q_rank``, keys and values of all heads from one of width
    ``kv_rank``, and a rotated key part of ``rot_dim`` coordinates is shared by the heads; the latent and that part are what the
    cache keeps of a token. Per head ``dim`` unrotated and ``rot_dim`` rotated query / key coordinates and ``vdim`` values.
    ``rot`` turns the rotated part only."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    gate: str | None = None

    def __post_init__(self):
        if isinstance(self.rot, dict):
            object.__setattr__(self, "rot", RotarySpec(**self.rot))
        if self.rot.dims != self.rot_dim:
            raise ValueError(f"a rotation of {self.rot.dims} coordinates of a rotated part of {self.rot_dim}")
        if self.gate not in (None, "channel"):
            raise ValueError(f"latent attention has no gate {self.gate!r}")

    @property
    def kv_heads(self) -> int:
        return self.heads  # every head expands keys and values of its own

    @property
    def cached(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def gate_rows(self) -> int:
        return _gate_rows(self.gate, self.heads, self.vdim)

    def cache_geometry(self, tp: int = 1) -> tuple[int, int, int]:
        return 1, self.cached, 0

    def params(self, width: int) -> int:
        n = width * (self.q_rank + self.cached + self.gate_rows + self.heads * self.vdim) + self.q_rank + self.kv_rank
        return n + self.heads * ((self.dim + self.rot_dim) * self.q_rank + (self.dim + self.vdim) * self.kv_rank)


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule. Per head a state S [dim, vdim] follows ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q``; q, k and
    v come from a causal convolution over ``conv`` tokens per channel and silu, q and k as unit vectors (q times dim^-1/2).
    ``decay``: g = exp(-exp(A_log) softplus(projection + dt_bias)) is one number per "head" or one per key "channel".
    The output is RMS normed per head and multiplied by ``gate``(projection). ``decay_rank`` / ``gate_rank``: inner width
    of a two-factor projection (None: one full matrix)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay: str = "head"
    gate: str = "silu"
    decay_rank: int | None = None
    gate_rank: int | None = None

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads do not divide over {self.kv_heads} query/key heads")
        if self.decay not in ("head", "channel") or self.gate not in ("silu", "sigmoid"):
            raise ValueError(f"unknown decay {self.decay!r} or gate {self.gate!r}")
        if self.conv < 1:
            raise ValueError(f"a convolution over {self.conv} tokens")

    @property
    def decays(self) -> int:
        """Decay factors of one token."""
        return self.heads * (self.dim if self.decay == "channel" else 1)

    @property
    def channels(self) -> int:
        """Channels that pass the convolution: q, k, v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def params(self, width: int) -> int:
        pair = lambda n, r: n * width if r is None else r * (width + n)  # noqa: E731
        n = self.channels * (width + self.conv) + self.heads * (width + 1) + self.decays + self.vdim
        return n + pair(self.decays, self.decay_rank) + pair(self.heads * self.vdim, self.gate_rank) + width * self.heads * self.vdim


@dataclass(frozen=True)
class StateSpaceSpec:
    """State-space duality (Mamba-2). Per head a state S [dim, vdim] follows ``S <- exp(-exp(A_log) dt) S + dt B x^T``, ``y = S^T C + D x`` with
    ``dt = softplus(projection + dt_bias)``; B and C belong to groups of heads; x, B and C come from a causal convolution (with bias)
    over ``conv`` tokens per channel and silu. The heads' outputs times silu of a gate are RMS normed in ``norm_groups`` equal parts."""

    heads: int
    groups: int
    dim: int
    vdim: int
    conv: int
    norm_groups: int = 1

    def __post_init__(self):
        if self.groups < 1 or self.heads % self.groups:
            raise ValueError(f"{self.heads} heads do not divide over {self.groups} groups")
        if self.conv < 1:
            raise ValueError(f"a convolution over {self.conv} tokens")
        if self.norm_groups < 1 or (self.heads * self.vdim) % self.norm_groups:
            raise ValueError(f"{self.heads} x {self.vdim} channels do not divide into {self.norm_groups} normed parts")

    @property
    def kv_heads(self) -> int:
        return self.groups

    @property
    def channels(self) -> int:
        """Channels that pass the convolution: x, B, C."""
        return self.heads * self.vdim + 2 * self.groups * self.dim

    def params(self, width: int) -> int:
        inner = self.heads * self.vdim
        return width * (2 * inner + self.channels + self.heads) + self.channels * (self.conv + 1) + 3 * self.heads + inner


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Matrix memory with exponential gates (the mLSTM of xLSTM). Per head a state S [dim, vdim] and a normaliser n [dim] follow, with log
    gates i and f capped softly at ``gate_cap`` and a running maximum m that keeps the exponentials in range,
    ``S <- exp(f + m' - m) S + exp(i - m) k v^T`` (n alike), ``o = S^T q / (max(|n q|, exp(-m)) + 1e-6)``. The output is RMS normed per head
    with a weight per channel and multiplied by a sigmoid gate."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def __post_init__(self):
        if not self.gate_cap > 0:
            raise ValueError(f"gates capped at {self.gate_cap}")

    @property
    def kv_heads(self) -> int:
        return self.heads

    def params(self, width: int) -> int:
        inner = self.heads * self.vdim
        return width * (2 * self.heads * self.dim + 3 * inner + 2 * self.heads) + inner + 2 * self.heads


RECURRENT = (DeltaSpec, StateSpaceSpec, MatrixMemorySpec)  # mixers that keep a state per request instead of keys and values
Mixer = AttentionSpec | LatentSpec | DeltaSpec | StateSpaceSpec | MatrixMemorySpec


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same input; the result is ``left_scale * left + right_scale * right``."""

    left: Mixer
    right: Mixer
    left_scale: float = 1.0
    right_scale: float = 1.0

    def __post_init__(self):
        if any(getattr(m, "vo_bias", False) or getattr(m, "kv_from", None) is not None for m in (self.left, self.right)):
            raise ValueError("mixers side by side have neither output biases nor another layer's keys and values")

    def params(self, width: int) -> int:
        return self.left.params(width) + self.right.params(width)


def _mixer_of(x):
    if not isinstance(x, dict):
        return x
    if "left" in x:
        return ParallelSpec(**{**x, "left": _mixer_of(x["left"]), "right": _mixer_of(x["right"])})
    kinds = (("norm_groups", StateSpaceSpec), ("gate_cap", MatrixMemorySpec), ("conv", DeltaSpec), ("kv_rank", LatentSpec))
    return next((kind for key, kind in kinds if key in x), AttentionSpec)(**x)


@dataclass(frozen=True)
class FeedForwardSpec:
    """Dense (``experts`` None) or mixture-of-experts feed-forward. ``gated``: ``down(act(gate x) * up x)``, otherwise
    ``down(act(up x))``; with experts the same form is every expert's. ``score`` / ``renorm``: router scores over all
    experts, kept as they are or divided by the sum of the chosen ones. ``shared_ff`` > 0: an expert of that width runs
    for every token, scaled by a sigmoid gate of its own when ``shared_gate``. ``router_bias``: added to the router's logits.
    ``score`` "softmax" or "sigmoid". ``expert_groups`` > 1: the experts form that many groups of neighbours, a group's score is the sum of
    its two best ones, and only experts of the ``keep_groups`` best groups can be chosen. ``act`` "poly_norm": ``a N(z) + b N(z^2) + c N(z^3)
    + e`` of the row's hidden units with learned numbers, N dividing a row by its root mean square."""

    ff: int
    act: str
    gated: bool = True
    experts: int | None = None
    top: int = 1
    score: str = "softmax"
    renorm: bool = False
    shared_ff: int = 0
    shared_gate: bool = False
    router_bias: bool = False
    expert_groups: int = 1
    keep_groups: int = 1

    def __post_init__(self):
        if self.act not in ("silu", "gelu_tanh", "relu2", "poly_norm"):
            raise ValueError(f"unknown activation {self.act!r}")
        if self.act == "poly_norm" and (self.gated or self.experts is not None):
            raise ValueError("a normed polynomial is the activation of dense, ungated feed-forwards")
        if self.score not in ("softmax", "sigmoid"):
            raise ValueError(f"unknown router score {self.score!r}")
        if self.expert_groups != 1 or self.keep_groups != 1:
            per, rest = divmod(self.experts or 0, self.expert_groups)
            if rest or not 1 <= self.keep_groups <= self.expert_groups or self.top > self.keep_groups * per:
                raise ValueError(f"{self.top} of {self.experts} experts in the best {self.keep_groups} of {self.expert_groups} groups")
            if self.score != "sigmoid":
                raise ValueError("groups of experts are compared by sigmoid scores")
        if self.experts is not None and not 1 <= self.top <= self.experts:
            raise ValueError(f"{self.top} of {self.experts} experts per token")

    def params(self, width: int) -> int:
        mats = 3 if self.gated else 2
        if self.experts is None:
            return mats * width * self.ff + (4 if self.act == "poly_norm" else 0)
        n = self.experts * (mats * width * self.ff + width + (1 if self.router_bias else 0))
        if self.shared_ff:
            n += mats * width * self.shared_ff + (width if self.shared_gate else 0)
        return n


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer | ParallelSpec
    mlp: FeedForwardSpec | None = None  # None: the layer is its mixer only
    parallel_ff: bool = False  # mixer and feed-forward read the same normed input and join the stream in one sum

    def __post_init__(self):
        m = self.mlp
        if self.parallel_ff and m is not None and m.experts is not None and m.shared_gate:
            raise ValueError("the shared expert of a mixture beside the mixer has no gate: its output is summed with the mixer's")
        if self.parallel_ff and m is not None and m.act == "poly_norm":
            raise ValueError("a normed polynomial is the activation of a feed-forward behind its mixer")

    @property
    def joint_ff(self) -> tuple[str, int] | None:
        """(stem of its tensors, width) of the dense feed-forward that is computed together with the mixer: the whole one, or the
        shared expert of a mixture."""
        m = self.mlp
        if not self.parallel_ff or m is None:
            return None
        if m.experts is None:
            return "mlp", m.ff
        return ("mlp.shared", m.shared_ff) if m.shared_ff else None

    @classmethod
    def of(cls, x) -> "LayerSpec":
        """Accepts a ``LayerSpec`` or its ``dataclasses.asdict`` form (presets, argument namespaces read from JSON)."""
        if isinstance(x, cls):
            return x
        mlp = x.get("mlp")
        return cls(_mixer_of(x["mixer"]), mlp if mlp is None or isinstance(mlp, FeedForwardSpec) else FeedForwardSpec(**mlp),
                   x.get("parallel_ff", False))  # fmt: skip

    def to_dict(self) -> dict:
        return dataclasses.asdict(self)

    def branches(self) -> list[tuple[str, Mixer, float]]:
        """(prefix of its tensors behind ``l<i>.``, mixer, factor of its output) of every mixer of the layer."""
        m = self.mixer
        if isinstance(m, ParallelSpec):
            return [("mix.left.", m.left, m.left_scale), ("mix.right.", m.right, m.right_scale)]
        return [("mix.", m, 1.0)]

    def norms(self, post: bool) -> list[str]:
        """Names of the layer's norms: one per sub-layer, or with ``post`` two (of its input, and with a "b" of its output)."""
        subs = ["norm1"] if self.mlp is None or self.parallel_ff else ["norm1", "norm2"]
        return [n + x for n in subs for x in (("", "b") if post else ("",))]


def flat_sizes(specs: list[LayerSpec]) -> dict:
    """The ``ModelConfig`` size fields of a specified stack: the largest value of each over the layers."""
    mixers = [m for s in specs for _, m, _ in s.branches()]
    at = [m for m in mixers if isinstance(m, AttentionSpec)] or mixers
    ff = [s.mlp for s in specs if s.mlp is not None]
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


def pefolix_config(c: dict, shapes: dict | None = None) -> dict:
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


# ------------------------------------------------------------------------------------------------- Ledazen
# Fixed by the design: one norm per layer (RMS, weight stored around zero) whose output mixer and feed-forward both read,
# squared-relu feed-forward without a gate, rotation of interleaved pairs, q / k norms and a sink of score 0 in attention,
# the two forms of the delta rule (alone: a decay per head, silu gate; beside attention: a decay per key channel, sigmoid
# gate, both through two-factor projections), a bigram table added to the embedding.


def _rows_of(shapes: dict | None, name: str, m: dict, key: str) -> int:
    """Rows of a tensor that config.json need not state (the inner width of a two-factor projection, distance buckets): the
    checkpoint's tensor says it, or ``key`` of the mixer's description."""
    if shapes and name in shapes:
        return int(shapes[name][0])
    if key in m:
        return int(m[key])
    raise ValueError(f"the inner width of {name} (its rows) is not in config.json: give the checkpoint's tensor shapes, or {key!r} in the mixer")


def ledazen_config(c: dict, shapes: dict | None = None) -> dict:
    """``config.json`` of a Ledazen model (and the shapes of its tensors by name) -> ``ModelConfig`` arguments."""
    sizes = lambda m: (m["heads"], m["kv_heads"], m["dim"], m["vdim"])  # noqa: E731
    specs = []
    for i, layer in enumerate(c["layers"]):
        m, f = layer["mixer"], layer.get("mlp")
        if layer["type"] == "delta":
            mixer = DeltaSpec(*sizes(m), m["conv"])
        elif layer["type"] == "parallel":
            a, d = m["left"], m["right"]
            rot = RotarySpec(a["rot"]["dims"], float(a["rot"]["base"])) if a.get("rot") else None
            left = AttentionSpec(*sizes(a), float(a["scale"]), qk_norm=True, rot=rot, sink=0.0)
            p = f"l{i}.mix.right."
            right = DeltaSpec(*sizes(d), d["conv"], "channel", "sigmoid", _rows_of(shapes, p + "a1", d, "decay_rank"),
                              _rows_of(shapes, p + "g1", d, "gate_rank"))  # fmt: skip
            mixer = ParallelSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))
        else:
            raise ValueError(f"layer {i}: a Ledazen model has no mixer of type {layer['type']!r}")
        if f is not None and f["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        specs.append(LayerSpec(mixer, None if f is None else FeedForwardSpec(f["ff"], "relu2", gated=False), parallel_ff=True))
    b = c["embedding"]["bigram"]
    return dict(flat_sizes(specs), layer_specs=specs, hidden_size=c["width"], vocab_size=c["vocab"], norm_epsilon=c["norm"]["eps"],
                norm_offset=1.0, bigram=dict(buckets=b["buckets"], mul_prev=b["mul_prev"], mul_cur=b["mul_cur"]),
                tie_word_embeddings=False, model_arch="Ledazen")  # fmt: skip


def ledazen_json(cfg) -> dict:
    """The ``config.json`` of a Ledazen ``ModelConfig`` (inverse of ``ledazen_config``; carries the inner widths too)."""
    sizes = lambda m: dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim)  # noqa: E731
    layers = []
    for s in cfg.layer_specs:
        m = s.mixer
        if isinstance(m, DeltaSpec):
            kind, mixer = "delta", dict(sizes(m), conv=m.conv)
        else:
            left = dict(sizes(m.left), scale=m.left.scale)
            if m.left.rot is not None:
                left["rot"] = dict(dims=m.left.rot.dims, base=m.left.rot.base)
            right = dict(sizes(m.right), conv=m.right.conv, decay_rank=m.right.decay_rank, gate_rank=m.right.gate_rank)
            kind, mixer = "parallel", dict(left=left, right=right, left_scale=m.left_scale, right_scale=m.right_scale)
        layers.append(dict(type=kind, mixer=mixer, mlp=None if s.mlp is None else dict(kind="dense", ff=s.mlp.ff)))
    return dict(architecture="Ledazen", embedding=dict(bigram=dict(cfg.bigram)), layers=layers, norm=dict(eps=cfg.norm_epsilon),
                vocab=cfg.vocab_size, width=cfg.hidden_size)  # fmt: skip


# ------------------------------------------------------------------------------------------------- Zetizen
# Fixed by the design: one layer norm per layer whose output mixer and feed-forward both read, a normed embedding that is also
# the output matrix; three mixers: attention with a learned distance bias and capped scores, chunked attention with stretched
# rotation of halves, keys as values and a gate per head, latent attention with a gate per channel; norms over whole query and
# key projections; gated silu experts weighted by a softmax over the chosen logits, a shared one beside them.


def _yarn_of(r: dict) -> RotarySpec:
    s = r.get("scaling")
    return RotarySpec(r["dims"], float(r["base"]), False, None if s is None else YarnSpec(float(s["factor"]), s["original"], float(s["fast"]), float(s["slow"])))


def zetizen_config(c: dict, shapes: dict | None = None) -> dict:
    """``config.json`` of a Zetizen model (and the shapes of its tensors by name) -> ``ModelConfig`` arguments."""
    specs = []
    for i, layer in enumerate(c["layers"]):
        m, f = layer["mixer"], layer.get("mlp")
        if layer["type"] == "latent_attention":
            mixer = LatentSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), _yarn_of(m["rot"]), "channel")
        elif layer["type"] in ("attention", "attention_2"):
            sizes = (m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]))
            both = dict(softcap=float(m["softcap"]) if m.get("softcap") else None, qk_norm=True, norm_over="projection")
            if layer["type"] == "attention":
                rows = _rows_of(shapes, f"l{i}.mix.rel", m, "bias_rows")
                mixer = AttentionSpec(*sizes, distance_bias=DistanceBiasSpec(rows, m["bias_max"]), **both)
            else:
                mixer = AttentionSpec(*sizes, rot=_yarn_of(m["rot"]), chunk=m["mask"]["size"], qk_bias=True, tied_values=True, gate="head", **both)
        else:
            raise ValueError(f"layer {i}: a Zetizen model has no mixer of type {layer['type']!r}")
        if f is not None and f["kind"] != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        mlp = None
        if f is not None:
            shared = f.get("shared")
            mlp = FeedForwardSpec(f["expert"]["ff"], "silu", experts=f["router"]["experts"], top=f["router"]["top"], renorm=True,
                                  shared_ff=shared["ff"] if shared else 0, router_bias=True)  # fmt: skip
        specs.append(LayerSpec(mixer, mlp, parallel_ff=True))
    return dict(flat_sizes(specs), layer_specs=specs, hidden_size=c["width"], vocab_size=c["vocab"], norm_epsilon=c["norm"]["eps"],
                norm_kind="layer", embed_norm=True, logit_scale=float(c["logit_scale"]), tie_word_embeddings=True, model_arch="Zetizen")  # fmt: skip


def zetizen_json(cfg) -> dict:
    """The ``config.json`` of a Zetizen ``ModelConfig`` (inverse of ``zetizen_config``; carries the number of distance buckets too)."""

    def rot(r: RotarySpec) -> dict:
        return dict(dims=r.dims, base=r.base, **({"scaling": dataclasses.asdict(r.scaling)} if r.scaling else {}))

    layers = []
    for s in cfg.layer_specs:
        a, f = s.mixer, s.mlp
        if isinstance(a, LatentSpec):
            kind, mixer = "latent_attention", dict(heads=a.heads, dim=a.dim, rot_dim=a.rot_dim, vdim=a.vdim, q_rank=a.q_rank, kv_rank=a.kv_rank,
                                                   scale=a.scale, rot=rot(a.rot))  # fmt: skip
        else:
            mixer = dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, softcap=a.softcap)
            if a.learned_bias is not None:
                kind, mixer = "attention", dict(mixer, bias_max=a.learned_bias.far, bias_rows=a.learned_bias.rows)
            else:
                kind, mixer = "attention_2", dict(mixer, mask=dict(size=a.chunk), rot=rot(a.rot))
        mlp = None
        if f is not None:
            mlp = dict(kind="moe", expert=dict(ff=f.ff), router=dict(experts=f.experts, top=f.top))
            if f.shared_ff:
                mlp["shared"] = dict(ff=f.shared_ff)
        layers.append(dict(type=kind, mixer=mixer, mlp=mlp))
    return dict(architecture="Zetizen", layers=layers, logit_scale=cfg.logit_scale, norm=dict(eps=cfg.norm_epsilon), vocab=cfg.vocab_size,
                width=cfg.hidden_size)  # fmt: skip


# ------------------------------------------------------------------------------------------------- Pebodra
# Fixed by the design: a norm (RMS, in parts) on every sub-layer's output and none on its input; three mixers: windowed
# differential attention with biases and norms of query and key halves, whose keys and values another layer may share;
# Mamba-2; mLSTM; dense feed-forwards with a normed polynomial, gated silu experts weighted by the sigmoid of their logits.


def pebodra_config(c: dict, shapes: dict | None = None) -> dict:
    """``config.json`` of a Pebodra model -> ``ModelConfig`` arguments."""
    specs = []
    for i, layer in enumerate(c["layers"]):
        m, f = layer["mixer"], layer.get("mlp")
        if layer["type"] == "attention":
            rot, mask = m.get("rot"), m.get("mask") or {}
            mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), mask.get("size"), qk_norm=True,
                                  rot=RotarySpec(rot["dims"], float(rot["base"]), False) if rot else None, qk_bias=True, vo_bias=True,
                                  diff=float(m["diff"]), kv_from=m.get("kv_from"))  # fmt: skip
        elif layer["type"] == "mamba2":
            mixer = StateSpaceSpec(m["heads"], m["groups"], m["state"], m["vdim"], m["conv"], m["norm_groups"])
        elif layer["type"] == "mlstm":
            mixer = MatrixMemorySpec(m["heads"], m["dim"], m["vdim"], float(m["gate_cap"]))
        else:
            raise ValueError(f"layer {i}: a Pebodra model has no mixer of type {layer['type']!r}")
        mlp = None
        if f is not None and f["kind"] == "dense":
            mlp = FeedForwardSpec(f["ff"], "poly_norm", gated=False)
        elif f is not None and f["kind"] == "moe":
            r = f["router"]
            g = r.get("groups") or dict(count=1, keep=1)
            mlp = FeedForwardSpec(f["expert"]["ff"], "silu", experts=r["experts"], top=r["top"], score="sigmoid", expert_groups=g["count"],
                                  keep_groups=g["keep"])  # fmt: skip
        elif f is not None:
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        specs.append(LayerSpec(mixer, mlp))
    return dict(flat_sizes(specs), layer_specs=specs, hidden_size=c["width"], vocab_size=c["vocab"], norm_epsilon=c["norm"]["eps"],
                norm_groups=c["norm"].get("groups") or 1, pre_norm=False, post_self_attn_layernorm=True, post_mlp_layernorm=True,
                logit_softcap=float(c["logit_softcap"]) if c.get("logit_softcap") else None, tie_word_embeddings=False,
                model_arch="Pebodra")  # fmt: skip


def pebodra_json(cfg) -> dict:
    """The ``config.json`` of a Pebodra ``ModelConfig`` (inverse of ``pebodra_config``)."""
    layers = []
    for s in cfg.layer_specs:
        a, f = s.mixer, s.mlp
        if isinstance(a, StateSpaceSpec):
            kind, mixer = "mamba2", dict(heads=a.heads, groups=a.groups, state=a.dim, vdim=a.vdim, conv=a.conv, norm_groups=a.norm_groups)
        elif isinstance(a, MatrixMemorySpec):
            kind, mixer = "mlstm", dict(heads=a.heads, dim=a.dim, vdim=a.vdim, gate_cap=a.gate_cap)
        else:
            kind, mixer = "attention", dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, diff=a.diff)
            if a.window is not None:
                mixer["mask"] = dict(size=a.window)
            if a.rot is not None:
                mixer["rot"] = dict(dims=a.rot.dims, base=a.rot.base)
            if a.kv_from is not None:
                mixer["kv_from"] = a.kv_from
        mlp = None
        if f is not None and f.experts is None:
            mlp = dict(kind="dense", ff=f.ff)
        elif f is not None:
            mlp = dict(kind="moe", expert=dict(ff=f.ff), router=dict(experts=f.experts, top=f.top, groups=dict(count=f.expert_groups, keep=f.keep_groups)))
        layers.append(dict(type=kind, mixer=mixer, mlp=mlp))
    return dict(architecture="Pebodra", layers=layers, logit_softcap=cfg.logit_softcap, norm=dict(eps=cfg.norm_epsilon, groups=cfg.norm_groups),
                vocab=cfg.vocab_size, width=cfg.hidden_size)  # fmt: skip


# ``config.json`` files that name their design in "architecture": name -> (reader(config, tensor shapes or None), writer)
LAYERED_ARCHITECTURES = {"Pefolix": (pefolix_config, pefolix_json), "Ledazen": (ledazen_config, ledazen_json),
                         "Zetizen": (zetizen_config, zetizen_json), "Pebodra": (pebodra_config, pebodra_json)}  # fmt: skip

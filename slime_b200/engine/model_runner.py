"""Rollout-engine model execution: weight buffers, prefill (extend) and decode forward passes.

Weights live in fused per-layer buffers ([q|k|v] rows, [gate;up] rows) sharded for the engine's
own TP degree; ``load_weights`` accepts Hugging Face tensor names (``q_proj``, ``gate_proj``, ...)
and stacks them into the fused buffers, so the trainer->engine sync contract is "HF names on the
wire" exactly as with the reference's engines. The same sm_100a kernels as the trainer are used
(RMSNorm with fused residual, RoPE(+QK-norm), SwiGLU, tcgen05 GEMM), so train and rollout
log-probs agree by construction. Decode runs under CUDA graphs per batch-size bucket.
"""

from __future__ import annotations

import logging
import math
import re

import torch

from slime_b200 import ops
from slime_b200.engine.kv_cache import PagedKVCache
from slime_b200.engine.projections import LayerProjections
from slime_b200.engine.state_cache import RecurrentStates, StateShape
from slime_b200.models.config import ModelConfig
from slime_b200.models.layer_spec import RECURRENT, AttentionSpec, DeltaSpec, LatentSpec, MatrixMemorySpec, StateSpaceSpec
from slime_b200.ops import delta, latent, linear_scan, stream, window_attention

logger = logging.getLogger(__name__)

_LAYER_RE = re.compile(r"^model\.layers\.(\d+)\.(.+)$")
_LAYERED_RE = re.compile(r"^l(\d+)\.(.+)$")  # designs described layer by layer (models/layer_spec.py)
_LAYERED_TOP = {"embed": "model.embed_tokens.weight", "head": "lm_head.weight", "final.norm": "model.norm.weight"}
_NORMS = {"norm1": "ln1", "norm1b": "post_attn_ln", "norm2": "ln2", "norm2b": "post_mlp_ln"}  # of a specified layer
_OUTPUT_NORMS = {"norm1": "post_attn_ln", "norm2": "post_mlp_ln"}  # where sub-layers read the stream itself
_MIMO_DRAFT_RE = re.compile(r"^model\.mtp_layers\.(\d+)\.(.+)$")


KV_KINDS = ("attention", "mla")  # layer kinds that keep keys and values in the paged cache


def cached_mixers(L) -> list[AttentionSpec | LatentSpec | None]:
    """What layer ``L`` keeps keys and values for: the attention mixers of a specified layer (but not those that use another
    layer's), one unnamed entry of another attention layer, nothing for a recurrent one."""
    if L["kind"] == "specified":
        return [m for _, m, _ in L["spec"].branches() if not isinstance(m, RECURRENT) and getattr(m, "kv_from", None) is None]
    return [None] if L["kind"] in KV_KINDS else []


class EngineWeights:
    """Fused, TP-sharded weight buffers addressed by Hugging Face names."""

    def __init__(self, cfg: ModelConfig, dtype, device, tp_size=1, tp_rank=0, ep_size=1, quantization: str | None = None,
                 draft_layers: int = 0):
        """``draft_layers``: how many multi-token-prediction depths (checkpoint layers ``num_layers + k``) to keep for
        speculative decoding; 0 ignores them.
        ``quantization="fp8"`` keeps the projection matrices whose shapes allow it as block-scaled e4m3
        (``engine/quant.py``); embeddings, the LM head, routers, norms and biases stay in ``dtype``.
        ``ep_size`` is 1 (every rank holds all experts and computes all routes) or ``tp_size`` (rank r holds experts
        ``r*E/ep ... (r+1)*E/ep - 1`` at full width; the ranks' expert outputs are summed like any row-parallel
        projection). Same split as ``--sglang-ep-size`` with the all-reduce MoE path (scripts/models/qwen3-30B-A3B.sh and
        tests/test_qwen3_30B_A3B.py:98-120 in the reference run rollout engines with ep 8)."""
        self.cfg, self.dtype, self.device, self.tp, self.rank = cfg, dtype, device, tp_size, tp_rank
        if ep_size not in (1, tp_size):
            raise ValueError(f"engine expert parallelism must be 1 or the engine's size ({tp_size}), got {ep_size}")
        self.ep = ep_size
        if cfg.num_experts is not None and cfg.num_experts % ep_size:
            raise ValueError(f"{cfg.num_experts} experts do not divide over {ep_size} ranks")
        self.experts_local = None if cfg.num_experts is None else cfg.num_experts // ep_size
        self.first_expert = 0 if cfg.num_experts is None or ep_size == 1 else tp_rank * self.experts_local
        h, d = cfg.hidden_size, cfg.head_dim
        self.hq, self.hkv = cfg.num_attention_heads // tp_size, max(cfg.num_query_groups // tp_size, 1)
        self.f = cfg.ffn_hidden_size // tp_size
        self.vocab_local = cfg.padded_vocab_size // tp_size
        e = lambda *s: torch.zeros(*s, dtype=dtype, device=device)  # noqa: E731
        if quantization not in (None, "fp8"):
            raise ValueError(f"unknown engine quantization {quantization!r} (None or 'fp8')")
        self.quantization = quantization

        def mat(*shape, parts=()):
            """A projection matrix: fp8 when asked for and every separately loaded row range starts on a scale block."""
            from slime_b200.engine import quant

            if quantization == "fp8" and quant.supported(shape[-2], shape[-1], parts):
                return quant.Fp8Weight(*shape, device=device)
            return e(*shape)

        self.vision = None  # image encoder, replicated on every rank of the engine
        if cfg.vision is not None:
            from slime_b200.models.vision import VisionConfig, VisionTower

            self.vision = VisionTower(VisionConfig.from_dict(cfg.vision), dtype, device).requires_grad_(False)
        self.embed = e(self.vocab_local, h)
        self.lm_head = self.embed if cfg.tie_word_embeddings else e(self.vocab_local, h)
        self.final_norm = e(h)
        self.embed_norm = e(h) if cfg.embed_norm else None
        self.bigram = e(cfg.bigram["buckets"] + 1, h) if cfg.bigram else None  # replicated over tensor-parallel ranks
        self._specified_tensors = None
        self.layers = []
        self.draft = []  # draft heads: an ordinary layer plus the two input norms, the joining projection and a final norm
        self.num_draft_layers = draft_layers
        for i in range(cfg.num_layers + draft_layers):
            kind = cfg.mixer(i)
            if kind == "specified":
                self.layers.append(self._specified_buffers(cfg.layer_specs[i], e, mat))
                continue
            if kind not in ("attention", "general_attention", "gated_delta_net", "mla", "dsa"):
                raise NotImplementedError(f"the rollout engine has no layer of kind {kind!r} (layer {i})")
            full_norm = cfg.qk_layernorm_full  # one weight per projection (sharded like it) instead of one per head
            if kind == "gated_delta_net":
                # linear-attention layer: replicated over tensor-parallel ranks (every rank computes all of it)
                kd, vd = cfg.linear_num_key_heads * cfg.linear_key_head_dim, cfg.linear_num_value_heads * cfg.linear_value_head_dim
                hv = cfg.linear_num_value_heads
                f32 = lambda *sh: torch.zeros(*sh, dtype=torch.float32, device=device)  # noqa: E731
                L = {"kind": "gdn", "ln1": e(h), "ln2": e(h), "post_attn_ln": None, "post_mlp_ln": None,
                     "gdn_conv": e(2 * kd + vd, cfg.linear_conv_kernel_dim), "gdn_dt_bias": f32(hv), "gdn_A_log": f32(hv),
                     "gdn_norm": e(cfg.linear_value_head_dim), "gdn_out": e(h, vd)}  # fmt: skip
                if "qwen3next" in (cfg.model_arch or "").lower().replace("_", ""):
                    L.update(gdn_qkvz=e(2 * kd + 2 * vd, h), gdn_ba=e(2 * hv, h))
                else:
                    L.update(gdn_qkv=e(2 * kd + vd, h), gdn_z=e(vd, h), gdn_b=e(hv, h), gdn_a=e(hv, h))
            elif kind in ("mla", "dsa"):
                # latent attention: the compressions are replicated, the per-head expansions are sharded by head
                hq_l, dn, dr, dv = cfg.num_attention_heads // tp_size, cfg.qk_head_dim, cfg.qk_pos_emb_head_dim, cfg.v_head_dim
                L = {"kind": "mla", "ln1": e(h), "ln2": e(h), "post_attn_ln": None, "post_mlp_ln": None,
                     "kv_a": e(cfg.kv_lora_rank + dr, h), "kv_a_ln": e(cfg.kv_lora_rank), "kv_b": e(hq_l * (dn + dv), cfg.kv_lora_rank),
                     "o": e(h, hq_l * dv)}  # fmt: skip
                if cfg.q_lora_rank:
                    L.update(q_a=e(cfg.q_lora_rank, h), q_a_ln=e(cfg.q_lora_rank), q_b=e(hq_l * (dn + dr), cfg.q_lora_rank))
                else:
                    L["q_proj"] = e(hq_l * (dn + dr), h)
                if kind == "dsa":
                    # lightning indexer (replicated): which cached tokens a query may attend; a layer for which
                    # max(layer - offset, 0) % freq != 0 (1-based) reuses the choice of the nearest earlier computing layer
                    one_based = i + 1
                    src = one_based
                    while (max(src - cfg.index_skip_topk_offset, 0) % cfg.index_topk_freq) != 0:
                        src -= 1
                    L["index_source"] = src - 1
                    if src == one_based:
                        hi, di = cfg.index_n_heads, cfg.index_head_dim
                        L.update(idx_wq_b=e(hi * di, cfg.q_lora_rank), idx_wk=e(di, h), idx_k_norm_w=e(di), idx_k_norm_b=e(di),
                                 idx_weights=e(hi, h))  # fmt: skip
            else:
                L = self._attention_buffers(e, mat, h, d, full_norm)
            L.setdefault("kind", "attention")
            if cfg.is_moe_layer(i):
                el = self.experts_local
                fe = cfg.moe_ffn_hidden_size
                L.update(router=e(cfg.num_experts, h), w13=mat(el, 2 * fe, h, parts=(fe,)), w2=mat(el, h, fe))
                if cfg.moe_router_enable_expert_bias:
                    L["router_bias"] = torch.zeros(cfg.num_experts, dtype=torch.float32, device=device)
                if cfg.moe_shared_expert_intermediate_size:
                    fs = cfg.moe_shared_expert_intermediate_size // tp_size
                    L.update(shared_gate_up=mat(2 * fs, h, parts=(fs,)), shared_down=mat(h, fs))
                    if cfg.moe_shared_expert_gate:
                        L["shared_gate"] = e(1, h)
            else:
                L.update(gate_up=mat(2 * self.f, h, parts=(self.f,)), down=mat(h, self.f))
            if i >= cfg.num_layers:
                if L["kind"] == "gdn" or kind == "dsa":
                    raise NotImplementedError(f"a draft head with a {kind} mixer is not supported by the rollout engine")
                L.update(enorm=e(h), hnorm=e(h), eh_proj=e(h, 2 * h), final_ln=e(h))
                self.draft.append(L)
            else:
                self.layers.append(L)
        self.version = "default"

    def _attention_buffers(self, e, mat, h, d, full_norm):
        cfg = self.cfg
        L = {
            "ln1": e(h), "qkv": mat((self.hq + 2 * self.hkv) * d, h, parts=(self.hq * d, (self.hq + self.hkv) * d)),
            "o": mat(h, self.hq * d), "ln2": e(h),
            "qkv_bias": e((self.hq + 2 * self.hkv) * d) if cfg.add_qkv_bias else None,
            "q_norm": e(self.hq * d if full_norm else d) if (cfg.qk_layernorm or full_norm) else None,
            "k_norm": e(self.hkv * d if full_norm else d) if (cfg.qk_layernorm or full_norm) else None,
            "post_attn_ln": e(h) if cfg.post_self_attn_layernorm else None,
            "post_mlp_ln": e(h) if cfg.post_mlp_layernorm else None,
        }  # fmt: skip
        if cfg.attention_output_gate:
            L["gate"] = e(self.hq * d, h)  # sigmoid gate of the attention output, one row per query channel
        if cfg.softmax_sinks:
            L["sinks"] = torch.zeros(self.hq, dtype=torch.float32, device=self.device)  # per-head logit in the denominator
        return L

    def _specified_buffers(self, spec, e, mat) -> dict:
        """Buffers of a layer that has its own ``LayerSpec``: the fused matrices of ``LayerProjections``; for a feed-forward behind
        the mixer gate and up rows stacked, and the router's rows followed by the shared expert's gate (one product
        computes both; rows padded to a multiple of 8)."""
        h, m, tp = self.cfg.hidden_size, spec.mlp, self.tp
        if self.cfg.padded_vocab_size % tp:
            raise ValueError(f"a vocabulary of {self.cfg.padded_vocab_size} does not divide over {tp} tensor-parallel ranks")
        lay = LayerProjections(spec, tp)
        attention_only = not any(isinstance(x, RECURRENT) for _, x, _ in spec.branches())
        L = {"kind": "specified", "spec": spec, "proj": lay}
        L.update({self._norm_keys[n]: e(h) for n in self.cfg.spec_norms(spec)})
        # block-scaled fp8 covers plain attention projections; what enters a recurrence keeps its precision
        L["in"] = mat(lay.in_rows, h, parts=[r for r, _ in lay.ins.values() if r]) if attention_only else e(lay.in_rows, h)
        L["out"] = mat(h, lay.out_cols) if attention_only and len(lay.outs) == 1 else e(h, lay.out_cols)
        if lay.biased:
            L["in_bias"] = e(lay.in_rows)
        if lay.out_biased:
            L["out_bias"] = e(h)
        f32 = lambda *n: torch.zeros(*n, dtype=torch.float32, device=self.device)  # noqa: E731
        for p, x, _ in spec.branches():
            if isinstance(x, LatentSpec):
                n = x.heads // tp
                L.update({p + "dq.norm": e(x.q_rank), p + "dkv.norm": e(x.kv_rank), p + "up_q": mat(n * (x.dim + x.rot_dim), x.q_rank),
                          p + "up_kv": e(n * (x.dim + x.vdim), x.kv_rank)})  # fmt: skip
                continue
            if isinstance(x, DeltaSpec):
                L.update({p + "conv": e(x.channels // tp, x.conv), p + "A_log": f32(x.heads // tp), p + "dt_bias": f32(x.decays // tp),
                          p + "norm": e(x.vdim)})  # fmt: skip
                if p in lay.low:
                    L[p + "low"] = e(lay.low[p][2], lay.low[p][1])
                continue
            if isinstance(x, StateSpaceSpec):
                if x.norm_groups % tp:
                    raise ValueError(f"{x.norm_groups} normed parts do not divide over {tp} tensor-parallel ranks")
                L.update({p + "conv": e(x.channels // tp, x.conv), p + "conv.b": e(x.channels // tp), p + "norm": e(x.heads * x.vdim // tp)})
                L.update({p + n: f32(x.heads // tp) for n in ("A_log", "dt_bias", "D")})
                continue
            if isinstance(x, MatrixMemorySpec):
                L.update({p + "i.b": f32(x.heads // tp), p + "f.b": f32(x.heads // tp), p + "norm": e(x.heads * x.vdim // tp)})
                continue
            if x.qk_norm:
                whole = x.norm_over == "projection"  # sharded like the projections
                nq, nk = x.norm_widths()
                L[p + "q.norm"] = e(nq // tp if whole else nq)
                if x.kv_from is None:
                    L[p + "k.norm"] = e(nk // tp if whole else nk)
            if x.diff is not None:  # the vectors as stored, and the factor of the second attention they give
                L.update({p + "pair_rows": f32(4, x.dim), p + "pair": f32(1)})
            if x.learned_bias is not None:
                # the table as it is stored, and spread over distances: [distance, head], the last row for everything beyond
                rows = x.learned_bias.by_distance()
                L.update({p + "rel": e(x.learned_bias.rows, x.heads // tp), p + "rel_rows": torch.tensor(rows, device=self.device),
                          p + "bias": f32(len(rows), x.heads // tp)})  # fmt: skip
        if m is None or (spec.parallel_ff and m.experts is None):
            return L
        up = 2 if m.gated else 1
        if m.experts is None:
            if m.ff % tp:
                raise ValueError(f"a feed-forward of width {m.ff} does not divide over {tp} tensor-parallel ranks")
            f = m.ff // tp
            L.update(gate_up=mat(up * f, h, parts=(f,)), down=mat(h, f))
            if m.act == "poly_norm":
                L["act_coef"] = f32(4)
            return L
        if m.experts % self.ep or (m.shared_ff % tp and not spec.parallel_ff):
            raise ValueError(f"{m.experts} experts / a shared expert of width {m.shared_ff} do not divide over {tp} ranks")
        el, fs = m.experts // self.ep, m.shared_ff // tp
        L.update(first_expert=0 if self.ep == 1 else self.rank * el, router=e(-(-(m.experts + 1) // 8) * 8, h),
                 w13=mat(el, up * m.ff, h, parts=(m.ff,)), w2=mat(el, h, m.ff))  # fmt: skip
        if m.router_bias:
            L["router_shift"] = f32(m.experts)
        if m.shared_ff and not spec.parallel_ff:
            L.update(shared_gate_up=mat(up * fs, h, parts=(fs,)), shared_down=mat(h, fs))
        return L

    def specified_tensors(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint tensors (name -> full shape) of a model with ``layer_specs``."""
        if self._specified_tensors is None:
            h, v = self.cfg.hidden_size, self.cfg.vocab_size
            out = {"embed": (v, h), "final.norm": (h,)}
            if not self.cfg.tie_word_embeddings:
                out["head"] = (v, h)
            if self.cfg.embed_norm:
                out["embed.norm"] = (h,)
            if self.cfg.bigram:
                out["bigram"] = (self.cfg.bigram["buckets"] + 1, h)
            for i, s in enumerate(self.cfg.layer_specs):
                m, p = s.mlp, f"l{i}."
                out.update({p + n: (h,) for n in self.cfg.spec_norms(s)})
                out.update({p + n: shape for n, shape in LayerProjections(s).tensors(h).items()})
                if m is None or (s.parallel_ff and m.experts is None):
                    continue
                stems = {p + "mlp": m.ff}
                if m.experts is not None:
                    stems = {f"{p}mlp.e{e}": m.ff for e in range(m.experts)}
                    out[p + "mlp.router"] = (m.experts, h)
                    if m.router_bias:
                        out[p + "mlp.router.b"] = (m.experts,)
                    if m.shared_ff and not s.parallel_ff:
                        stems[p + "mlp.shared"] = m.shared_ff
                    if m.shared_gate:
                        out[p + "mlp.shared.sg"] = (1, h)
                if m.act == "poly_norm":
                    out[p + "mlp.act"] = (4,)
                for stem, f in stems.items():
                    out.update({stem + ".up": (f, h), stem + ".down": (h, f)})
                    if m.gated:
                        out[stem + ".gate"] = (f, h)
            self._specified_tensors = out
        return self._specified_tensors

    def _load_mixer(self, L, sub: str, t, raw) -> bool:
        """A tensor of a specified layer's mixers, or of a feed-forward beside them; False when it is neither."""
        lay, h = L["proj"], self.cfg.hidden_size
        if sub in lay.ins:
            r0, rows = lay.ins[sub]
            self._put(L["in"], r0, rows, None if sub in lay.whole else 0, t, raw, scale=False)
            return True
        if sub in lay.split:  # several projections in one tensor
            parts = lay.split[sub]
            for (name, _), part in zip(parts, t.split([rows for _, rows in parts])):
                self._put(L["in"], *lay.ins[name], 0, part, part, scale=False)
            return True
        if sub.endswith(".b") and sub[:-2] in lay.out_biased:
            if self.rank == 0:  # the ranks' outputs are summed
                L["out_bias"].copy_(t)
            return True
        if sub in lay.outs:
            c0, cols = lay.outs[sub]
            if isinstance(L["out"], torch.Tensor):
                L["out"][:, c0 : c0 + cols].copy_(t[:, self.rank * cols : (self.rank + 1) * cols])
            else:
                self._put(L["out"], 0, h, 1, t, raw, scale=False)
            return True
        if sub.endswith(".b") and sub[:-2] in lay.biased:
            r0, rows = lay.ins[sub[:-2]]
            L["in_bias"][r0 : r0 + rows].copy_(self._rows(t, rows))
            return True
        for p, (_, _, _, parts) in lay.low.items():
            if sub in parts:
                r0, rows, c0, cols = parts[sub]
                L[p + "low"][r0 : r0 + rows, c0 : c0 + cols].copy_(self._rows(t, rows))
                return True
        for p, m, _ in L["spec"].branches():
            if isinstance(m, LatentSpec):
                n = m.heads // self.tp
                if sub in (p + "dq.norm", p + "dkv.norm"):
                    L[sub].copy_(t)
                elif sub == p + "uq":
                    self._put(L[p + "up_q"], 0, n * (m.dim + m.rot_dim), 0, t, raw, scale=False)
                elif sub in (p + "uk", p + "uv"):
                    r0, rows = (0, n * m.dim) if sub == p + "uk" else (n * m.dim, n * m.vdim)
                    L[p + "up_kv"][r0 : r0 + rows].copy_(self._rows(t, rows))
                else:
                    continue
                return True
            if isinstance(m, StateSpaceSpec) and sub in (p + "conv", p + "conv.b"):
                v, g = m.heads * m.vdim, m.groups * m.dim
                L[sub].copy_(torch.cat([self._rows(part, n // self.tp) for part, n in zip(t.split([v, g, g]), (v, g, g))]))
                return True
            if isinstance(m, (StateSpaceSpec, MatrixMemorySpec)) and sub in L and sub.startswith(p):
                L[sub].copy_(self._rows(raw, L[sub].numel()))
                return True
            vectors = [p + n for n in ("lq1", "lk1", "lq2", "lk2")]
            if p + "pair" in L and sub in vectors:
                L[p + "pair_rows"][vectors.index(sub)].copy_(raw)
                self._weigh_pair(L, p, m)
                return True
            if sub in (p + "q.conv", p + "k.conv", p + "v.conv"):
                g, v = m.kv_heads // self.tp * m.dim, m.heads // self.tp * m.vdim
                r0, rows = {"q": (0, g), "k": (g, g), "v": (2 * g, v)}[sub[len(p)]]
                L[p + "conv"][r0 : r0 + rows].copy_(self._rows(t, rows))
                return True
            if sub in (p + "A_log", p + "dt_bias"):
                L[sub].copy_(self._rows(raw, L[sub].numel()))
                return True
            if sub == p + "rel":
                L[sub].copy_(t[:, self.rank * L[sub].shape[1] : (self.rank + 1) * L[sub].shape[1]])
                self._spread_bias(L, p)
                return True
            if sub in (p + "norm", p + "q.norm", p + "k.norm"):
                L[sub].copy_(self._rows(t, L[sub].numel()) if L[sub].numel() != t.numel() else t)
                return True
        return False

    def _spread_bias(self, L, p: str):
        """The learned distance bias by distance, from its table by bucket (in place: captured graphs keep its address)."""
        L[p + "bias"].copy_(L[p + "rel"].float().index_select(0, L[p + "rel_rows"]))

    def _weigh_pair(self, L, p: str, m: AttentionSpec):
        """Factor of the second attention of a pair, from its vectors (in place: captured graphs keep its address)."""
        q1, k1, q2, k2 = L[p + "pair_rows"]
        L[p + "pair"].copy_(torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum()) + m.diff)

    @property
    def _norm_keys(self) -> dict[str, str]:
        return _NORMS if self.cfg.pre_norm else _OUTPUT_NORMS

    def _load_specified(self, L, sub: str, t, raw) -> bool:
        """One tensor of a specified layer, addressed by its name behind ``l<i>.`` (one of ``specified_tensors``)."""
        spec, h, tp = L["spec"], self.cfg.hidden_size, self.tp
        m = spec.mlp
        if sub in self._norm_keys:
            L[self._norm_keys[sub]].copy_(t)
            return True
        if self._load_mixer(L, sub, t, raw):
            return True
        table = {}
        if m.experts is None:
            if sub == "mlp.act":
                L["act_coef"].copy_(raw)
                return True
            f = m.ff // tp
            table = {"mlp.gate": ("gate_up", 0, f, 0), "mlp.up": ("gate_up", f if m.gated else 0, f, 0), "mlp.down": ("down", 0, h, 1)}
        else:
            if sub == "mlp.router":
                L["router"][: m.experts].copy_(t)
                return True
            if sub == "mlp.router.b":
                L["router_shift"].copy_(raw)
                return True
            if sub == "mlp.shared.sg":
                L["router"][m.experts].copy_(t.view(-1))
                return True
            fs = m.shared_ff // tp
            if m.shared_ff:
                table.update({"mlp.shared.gate": ("shared_gate_up", 0, fs, 0), "mlp.shared.up": ("shared_gate_up", fs if m.gated else 0, fs, 0),
                              "mlp.shared.down": ("shared_down", 0, h, 1)})  # fmt: skip
            em = re.match(r"^mlp\.e(\d+)\.(gate|up|down)$", sub)
            if em is not None:
                e, which = int(em.group(1)) - L["first_expert"], em.group(2)
                if not 0 <= e < L["w2"].shape[0]:
                    return True  # another rank's expert
                if which == "down":
                    self._put(L["w2"][e], 0, h, None, t, raw, scale=False)
                else:
                    self._put(L["w13"][e], m.ff if which == "up" and m.gated else 0, m.ff, None, t, raw, scale=False)
                return True
        key, r0, rows, cut = table[sub]
        self._put(L[key], r0, rows, cut, t, raw, scale=False)
        return True

    def state_geometry(self) -> list[StateShape]:
        """Shapes of the states of this rank's recurrent mixers, in layer order."""
        c, out = self.cfg, []
        for L in self.layers:
            if L["kind"] == "gdn":
                out.append(StateShape(c.linear_num_value_heads, c.linear_key_head_dim, c.linear_value_head_dim, *L["gdn_conv"].shape))
            for _, m, _ in L["spec"].branches() if L["kind"] == "specified" else ():
                if isinstance(m, MatrixMemorySpec):
                    out.append(StateShape(m.heads // self.tp, m.dim, m.vdim, normalised=True))
                elif isinstance(m, RECURRENT):
                    out.append(StateShape(m.heads // self.tp, m.dim, m.vdim, m.channels // self.tp, m.conv))
        return out

    def num_bytes(self) -> int:
        seen, total = set(), 0
        for t in self.tensors():
            if t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()
        return total

    def tensors(self):
        from slime_b200.engine.quant import Fp8Weight

        yield self.embed
        yield self.lm_head
        yield self.final_norm
        if self.bigram is not None:
            yield self.bigram
        if self.embed_norm is not None:
            yield self.embed_norm
        if self.vision is not None:
            yield from self.vision.parameters()
        for L in self.layers + self.draft:
            for v in L.values():
                if isinstance(v, torch.Tensor) and v.is_floating_point():
                    yield v
                elif isinstance(v, Fp8Weight):  # a quantised matrix: its bytes and its scales
                    yield from v.tensors()

    # -- loading -----------------------------------------------------------------------
    def _rows(self, t, n_local):
        """This TP rank's slice of a tensor sharded on dim 0."""
        return t[self.rank * n_local : (self.rank + 1) * n_local]

    def load_weight(self, name: str, t: torch.Tensor):
        cfg, d = self.cfg, self.cfg.head_dim
        if cfg.layer_specs is not None:
            want = self.specified_tensors().get(name)
            if want is None:
                return False
            if tuple(t.shape) != want:
                raise ValueError(f"{name} has shape {tuple(t.shape)}, this model's is {want}")
            m = _LAYERED_RE.match(name)
            if m is not None:
                return int(m.group(1)) < len(self.layers) and self._load_specified(
                    self.layers[int(m.group(1))], m.group(2), t.to(self.device, self.dtype, non_blocking=True), t)
            if name == "bigram":
                self.bigram.copy_(t.to(self.device, self.dtype))
                return True
            if name == "embed.norm":
                self.embed_norm.copy_(t.to(self.device, self.dtype))
                return True
            name = _LAYERED_TOP.get(name, name)
        if name.startswith("model.visual."):  # the image encoder keeps the checkpoint's parameter names
            if self.vision is None:
                return True
            target = dict(self.vision.named_parameters()).get(name[len("model.visual.") :])
            if target is None:
                return False
            target.data.copy_(t.to(self.device, target.dtype))
            return True
        if name.startswith("model.language_model."):  # checkpoints with a vision tower nest the language model
            name = "model." + name[len("model.language_model.") :]
        if name.endswith((".mlp.experts.gate_up_proj", ".mlp.experts.down_proj")):  # a layer's experts in one stacked tensor
            from slime_b200.weight_sync.convert import split_stacked_experts

            return all([self.load_weight(n, w) for n, w in split_stacked_experts(cfg, name, t)])
        if ".block_sparse_moe." in name:  # MiniMax-M2 spelling of the expert tensors
            from slime_b200.weight_sync.convert import family_name_to_generic

            name = family_name_to_generic(name)
        raw = t
        t = t.to(self.device, self.dtype, non_blocking=True)
        if name == "model.embed_tokens.weight":
            self.embed[: min(self.vocab_local, t.shape[0] - self.rank * self.vocab_local)].copy_(
                t[self.rank * self.vocab_local : (self.rank + 1) * self.vocab_local]
            )
            return True
        if name == "lm_head.weight":
            if not cfg.tie_word_embeddings:
                self.lm_head[: min(self.vocab_local, t.shape[0] - self.rank * self.vocab_local)].copy_(
                    t[self.rank * self.vocab_local : (self.rank + 1) * self.vocab_local]
                )
            return True
        from slime_b200.weight_sync import convert

        plus1 = 1.0 if convert._zero_centred(cfg) else 0.0  # Qwen3-Next / Qwen3.5 store their RMSNorm weights minus one
        if name == "model.norm.weight":
            self.final_norm.copy_(t + plus1)
            return True
        if name.startswith("mtp."):
            return True  # Qwen3-Next / Qwen3.5 draft block: their recurrent trunks are not speculated on, the block is not kept
        mimo = _MIMO_DRAFT_RE.match(name)
        if mimo is not None:
            # MiMo stores its draft head outside the layer list, the joining projection's halves as (hidden, embedding)
            depth, sub = int(mimo.group(1)), mimo.group(2)
            if depth >= len(self.draft):
                return True
            if sub == "input_proj.weight":
                h_half, e_half = t.chunk(2, dim=1)
                self.draft[depth]["eh_proj"].copy_(torch.cat([e_half, h_half], dim=1))
                return True
            own = {"token_layernorm.weight": "enorm.weight", "hidden_layernorm.weight": "hnorm.weight",
                   "final_layernorm.weight": "shared_head.norm.weight"}  # fmt: skip
            return self.load_weight(f"model.layers.{len(self.layers) + depth}.{own.get(sub, sub)}", raw)
        m = _LAYER_RE.match(name)
        if m is None:
            return False
        sub = m.group(2)
        if int(m.group(1)) >= len(self.layers):
            # a draft (multi-token-prediction) depth stored as an extra layer (DeepSeek-V3 layout): kept only when the
            # engine speculates; its copies of the embedding and the output head are the trunk's
            depth = int(m.group(1)) - len(self.layers)
            if depth >= len(self.draft) or sub in ("embed_tokens.weight", "shared_head.head.weight"):
                return True
            L = self.draft[depth]
            own = {"enorm.weight": "enorm", "hnorm.weight": "hnorm", "eh_proj.weight": "eh_proj", "shared_head.norm.weight": "final_ln"}
            if sub in own:
                L[own[sub]].copy_(t)
                return True
        else:
            L = self.layers[int(m.group(1))]
        hq, hkv = self.hq, self.hkv
        q_rows, kv_rows = hq * d, hkv * d
        if sub.startswith("linear_attn."):
            if L["kind"] != "gdn":
                return False
            inner = sub[len("linear_attn.") :]
            table = {"in_proj_qkvz.weight": "gdn_qkvz", "in_proj_ba.weight": "gdn_ba", "in_proj_qkv.weight": "gdn_qkv",
                     "in_proj_z.weight": "gdn_z", "in_proj_b.weight": "gdn_b", "in_proj_a.weight": "gdn_a", "conv1d.weight": "gdn_conv",
                     "dt_bias": "gdn_dt_bias", "A_log": "gdn_A_log", "norm.weight": "gdn_norm", "out_proj.weight": "gdn_out"}  # fmt: skip
            key = table.get(inner)
            if key is None or key not in L:
                return False
            src = raw.to(self.device, L[key].dtype)
            L[key].copy_(src.squeeze(1) if inner == "conv1d.weight" and src.dim() == 3 else src)
            return True
        if L["kind"] == "mla" and sub.startswith("self_attn."):
            inner = sub[len("self_attn.") :]
            hq_l, dn, dr, dv = cfg.num_attention_heads // self.tp, cfg.qk_head_dim, cfg.qk_pos_emb_head_dim, cfg.v_head_dim
            whole = {"q_a_proj.weight": "q_a", "q_a_layernorm.weight": "q_a_ln", "kv_a_proj_with_mqa.weight": "kv_a",
                     "kv_a_layernorm.weight": "kv_a_ln"}  # fmt: skip
            by_head = {"q_b_proj.weight": ("q_b", dn + dr), "q_proj.weight": ("q_proj", dn + dr), "kv_b_proj.weight": ("kv_b", dn + dv)}
            if inner in whole and whole[inner] in L:
                L[whole[inner]].copy_(t)
                return True
            if inner in by_head and by_head[inner][0] in L:
                key, per = by_head[inner]
                L[key].copy_(self._rows(t, hq_l * per))
                return True
            if inner == "o_proj.weight":
                L["o"].copy_(t[:, self.rank * hq_l * dv : (self.rank + 1) * hq_l * dv])
                return True
            indexer = {"indexer.wq_b.weight": "idx_wq_b", "indexer.wk.weight": "idx_wk", "indexer.k_norm.weight": "idx_k_norm_w",
                       "indexer.k_norm.bias": "idx_k_norm_b", "indexer.weights_proj.weight": "idx_weights"}  # fmt: skip
            if inner in indexer and indexer[inner] in L:
                L[indexer[inner]].copy_(t)
                return True
            return False
        if sub == "self_attn.q_proj.weight" and cfg.attention_output_gate and L["kind"] == "attention":
            # checkpoint rows are per head (query, gate): split them into the fused projection's q rows and the gate matrix
            x = t.view(cfg.num_attention_heads, 2 * d, -1)
            q_full, g_full = x[:, :d].reshape(-1, x.shape[-1]), x[:, d:].reshape(-1, x.shape[-1])
            L["qkv"][: hq * d].copy_(self._rows(q_full, hq * d))
            L["gate"].copy_(self._rows(g_full, hq * d))
            return True
        vectors = {
            "input_layernorm.weight": lambda: L["ln1"].copy_(t + plus1),
            "post_attention_layernorm.weight": lambda: L["ln2"].copy_(t + plus1),
            "self_attn.q_proj.bias": lambda: L["qkv_bias"][:q_rows].copy_(self._rows(t, q_rows)),
            "self_attn.k_proj.bias": lambda: L["qkv_bias"][q_rows : q_rows + kv_rows].copy_(self._rows(t, kv_rows)),
            "self_attn.v_proj.bias": lambda: L["qkv_bias"][q_rows + kv_rows :].copy_(self._rows(t, kv_rows)),
            "self_attn.qkv_proj.bias": lambda: L["qkv_bias"].copy_(t),
            "self_attn.q_norm.weight": lambda: L["q_norm"].copy_((self._rows(t, q_rows) if cfg.qk_layernorm_full else t) + plus1),
            "self_attn.k_norm.weight": lambda: L["k_norm"].copy_((self._rows(t, kv_rows) if cfg.qk_layernorm_full else t) + plus1),
            "mlp.gate.weight": lambda: L["router"].copy_(t),
            "post_self_attn_layernorm.weight": lambda: L["post_attn_ln"].copy_(t),
            "post_mlp_layernorm.weight": lambda: L["post_mlp_ln"].copy_(t),
            "mlp.gate.e_score_correction_bias": lambda: L["router_bias"].copy_(raw.to(self.device, torch.float32)),
            "mlp.shared_expert_gate.weight": lambda: L["shared_gate"].copy_(t),
            "self_attn.sinks": lambda: L["sinks"].copy_(self._rows(raw.to(self.device, torch.float32), hq)),
        }
        if sub in vectors and sub.split(".")[0] in ("post_self_attn_layernorm", "post_mlp_layernorm") and L.get(
                "post_attn_ln" if sub.startswith("post_self") else "post_mlp_ln") is None:
            return False
        if sub in vectors:
            vectors[sub]()
            return True
        # matrices: (buffer, first row in the buffer, rows there, how the incoming tensor is cut for this rank:
        # 0 = by rows, 1 = by columns, None = already this rank's)
        f = self.f
        matrices = {
            "self_attn.q_proj": ("qkv", 0, q_rows, 0), "self_attn.k_proj": ("qkv", q_rows, kv_rows, 0),
            "self_attn.v_proj": ("qkv", q_rows + kv_rows, kv_rows, 0), "self_attn.qkv_proj": ("qkv", 0, q_rows + 2 * kv_rows, None),
            "self_attn.o_proj": ("o", 0, cfg.hidden_size, 1), "mlp.gate_proj": ("gate_up", 0, f, 0),
            "mlp.up_proj": ("gate_up", f, f, 0), "mlp.gate_up_proj": ("gate_up", 0, 2 * f, None),
            "mlp.down_proj": ("down", 0, cfg.hidden_size, 1),
        }  # fmt: skip
        if cfg.moe_shared_expert_intermediate_size:
            fs = cfg.moe_shared_expert_intermediate_size // self.tp
            for prefix in ("mlp.shared_experts", "mlp.shared_expert"):
                matrices.update({f"{prefix}.gate_proj": ("shared_gate_up", 0, fs, 0), f"{prefix}.up_proj": ("shared_gate_up", fs, fs, 0),
                                 f"{prefix}.down_proj": ("shared_down", 0, cfg.hidden_size, 1)})  # fmt: skip
        stem, _, kind = sub.rpartition(".")
        buf = None
        if stem in matrices and kind in ("weight", "weight_scale_inv"):
            key, r0, rows, cut = matrices[stem]
            if key not in L:
                return False
            buf = L[key]
        else:
            em = re.match(r"^mlp\.experts\.(\d+)\.(gate_proj|up_proj|down_proj)$", stem)
            if em is None or kind not in ("weight", "weight_scale_inv") or "w13" not in L:
                return False
            e, which = int(em.group(1)) - self.first_expert, em.group(2)
            if not 0 <= e < self.experts_local:
                return True  # another rank's expert
            fe = cfg.moe_ffn_hidden_size
            buf = L["w13"][e] if which != "down_proj" else L["w2"][e]
            r0, rows, cut = (fe if which == "up_proj" else 0), (cfg.hidden_size if which == "down_proj" else fe), None
        self._put(buf, r0, rows, cut, t, raw, scale=kind == "weight_scale_inv")
        return True

    def _put(self, buf, r0: int, rows: int, cut, t, raw, scale: bool):
        """Write this rank's part of an incoming matrix (or of its block scales) into rows ``[r0, r0 + rows)`` of ``buf``."""
        from slime_b200.engine.quant import BLOCK, Fp8Weight

        fp8_in = raw.dtype == torch.float8_e4m3fn
        src = raw.to(self.device, non_blocking=True) if (scale or fp8_in) else t
        unit = BLOCK if scale else 1  # scale tensors count in blocks of 128 rows / columns
        if cut == 0:
            n = -(-rows // unit)
            src = src[self.rank * n : (self.rank + 1) * n]
        elif cut == 1:
            cols = buf.shape[-1] // unit
            src = src[:, self.rank * cols : (self.rank + 1) * cols]
        if isinstance(buf, Fp8Weight):
            if scale:
                buf.load_scale_rows(r0, src)
            else:
                buf.load_rows(r0, src)
            return
        if scale or fp8_in:
            raise ValueError("block-fp8 weights were sent to an engine that keeps this matrix in bf16; start it with "
                             "quantization='fp8' (and shapes that are multiples of 128) or send bf16 weights")
        buf[r0 : r0 + src.shape[0]].copy_(src)

    def load_weights(self, named_tensors, version: str | None = None):
        missing = [n for n, t in named_tensors if not self.load_weight(n, t)]
        if version is not None:
            self.version = version
        return missing

    def init_random(self, seed: int = 0, std: float = 0.02):
        from slime_b200.engine.quant import Fp8Weight

        g = torch.Generator(device=self.device).manual_seed(seed)
        quantised = [v for L in self.layers + self.draft for v in L.values() if isinstance(v, Fp8Weight)]
        skip = {t.data_ptr() for v in quantised for t in v.tensors()}
        for t in self.tensors():
            if t.data_ptr() in skip:
                continue
            if t.dim() == 1:
                t.fill_(1.0)
            else:
                t.copy_(torch.empty(t.shape, dtype=torch.float32, device=self.device).normal_(0, std, generator=g))
        for v in quantised:
            v.fill_random_(std, g)
        stream_norms = [self.final_norm] + [L[k] for L in self.layers for k in _NORMS.values() if L.get(k) is not None]
        for t in stream_norms if self.cfg.norm_offset else ():  # stored as the difference from the offset
            t.fill_(1.0 - self.cfg.norm_offset)
        for L in self.layers:
            for k, t in L.items():
                if k in ("in_bias", "out_bias", "router_shift"):
                    t.zero_()
                if k.endswith("pair_rows"):
                    p = k[: -len("pair_rows")]
                    self._weigh_pair(L, p, next(m for q, m, _ in L["spec"].branches() if q == p))
                if k.endswith("rel_rows"):
                    self._spread_bias(L, k[: -len("rel_rows")])
                if k.endswith("A_log"):  # the decay parameter of the delta rule must start in its valid range
                    t.copy_(torch.empty_like(t).uniform_(1e-3, 16.0, generator=g).log())
        for L in self.layers + self.draft:
            if L.get("qkv_bias") is not None:
                L["qkv_bias"].zero_()


def _linear(x, w, bias=None, out_dtype=None, out=None):
    """``x @ w^T`` for a bf16 matrix (tcgen05 bf16 GEMM) or a block-fp8 one (activation quantised here, fp8 GEMM)."""
    if isinstance(w, torch.Tensor):
        return ops.gemm(x, w, bias=bias, out_dtype=out_dtype, out=out)
    from slime_b200.engine import quant

    return quant.linear(x, w, bias=bias, out_dtype=out_dtype, out=out)


def _grouped_linear(x, w, lay):
    from slime_b200.ops import grouped

    if isinstance(w, torch.Tensor):
        return grouped.grouped_gemm(x, w, lay)
    return grouped.grouped_gemm_fp8(x, w.q, w.scale, lay, out_dtype=x.dtype)


class ModelRunner:
    def __init__(self, cfg: ModelConfig, weights: EngineWeights, kv: PagedKVCache, max_batch: int, max_context: int,
                 use_cuda_graph: bool = True, tp_group=None, states: RecurrentStates | None = None):  # fmt: skip
        """``states``: recurrent states of the live requests, for models whose weights have a ``state_geometry``."""
        self.cfg, self.w, self.kv, self.states = cfg, weights, kv, states
        self.recurrent = bool(weights.state_geometry())
        assert not self.recurrent or states is not None
        self.device = weights.device
        self.max_batch, self.max_context = max_batch, max_context
        self.max_pages_per_req = -(-max_context // kv.page_size)
        # head dims other than 64 / 128 fall back to attention written with plain ops, which reads lengths on the host
        self.layered = cfg.layer_specs is not None  # fp32 residual stream, layers described one by one
        self.use_cuda_graph = use_cuda_graph and self.device.type == "cuda" and (self.layered or (
            cfg.head_dim in (64, 128) and not cfg.multi_latent_attention and not cfg.softmax_sinks))  # fmt: skip
        self.tp_group = tp_group
        # Row-parallel projections (attention output, MLP down) leave their result in fp32 when no cross-rank sum
        # follows: the fused add+RMSNorm reads it unrounded, and a skinny decode GEMM with a long K can then be cut
        # into K slices that the epilogue sums with TMA reduce-add.
        self._proj_dtype = torch.float32 if (self.device.type == "cuda" and weights.tp == 1 and not ops.library_mode()) else None
        # Tensor-parallel decode: all-reduce + residual add + RMSNorm as one peer-memory kernel when the ranks share an
        # NVLink domain; otherwise NCCL all-reduce followed by the fused add+norm.
        self._fused_tp = None
        if tp_group is not None and weights.tp > 1 and self.device.type == "cuda" and not self.layered:
            from slime_b200.parallel import fused_tp

            if fused_tp.usable(weights.tp, self.device, cfg.hidden_size):
                try:
                    self._fused_tp = fused_tp.FusedAllReduceNorm(tp_group, max_batch, cfg.hidden_size, self.device)
                except Exception as e:  # noqa: BLE001
                    logger.warning("fused tensor-parallel all-reduce unavailable (%r): using NCCL", e)
        # KV slabs exist for the attention layers only; recurrent mixers keep a state per request (``states``)
        self.kv_of, self.state_of, n_attn, n_state = [], [], 0, 0  # per layer: number of its first slab / state
        for L in weights.layers + weights.draft:  # a draft head's layer number is num_layers + depth
            n = len(cached_mixers(L))
            r = sum(isinstance(m, RECURRENT) for _, m, _ in L["spec"].branches()) if L["kind"] == "specified" else int(L["kind"] == "gdn")
            self.kv_of.append(n_attn if n else None)
            self.state_of.append(n_state if r else None)
            n_attn, n_state = n_attn + n, n_state + r
        self.has_mla = any(L["kind"] == "mla" for L in weights.layers)
        self._dsa_masks: dict[int, torch.Tensor] = {}  # key choices of the indexer layers of the pass in flight
        self._composed_attention = cfg.rotary_percent < 1.0 or cfg.rotary_interleaved or cfg.qk_layernorm_full or bool(cfg.mrope_section)
        # vision inputs: decode positions are the token index plus a per-request offset (an image advances the position
        # by its larger grid side only), prefill positions are three streams
        self.rope_delta = torch.zeros(max_batch, dtype=torch.int32, device=self.device) if cfg.mrope_section else None
        self._mrope_axes = None
        rot = int(cfg.head_dim * cfg.rotary_percent) // 2 * 2
        self.rope = None if self.layered else ops.rope_table(cfg, max_context + 1, rot, self.device)
        # specified attention mixers, by layer and prefix: this rank's distance-penalty factors, scores of the column without a value
        self.slopes, self.sinks, self.rotary = {}, {}, {}
        for li, L in enumerate(weights.layers if self.layered else ()):
            for p, a, _ in L["spec"].branches():
                if isinstance(a, RECURRENT):
                    continue
                f32 = lambda x: torch.tensor(x, dtype=torch.float32, device=self.device)  # noqa: E731
                if a.rot is not None and a.rot.dims and a.rot not in self.rotary:
                    self.rotary[a.rot] = stream.rotary_table(max_context + 1, a.rot.dims, a.rot.base, self.device,
                                                             frequencies=a.rot.frequencies(), gain=a.rot.gain())  # fmt: skip
                if isinstance(a, LatentSpec):
                    continue
                n, sl = a.heads // weights.tp, a.slopes()
                self.slopes[li, p] = None if sl is None else f32(sl[weights.rank * n : (weights.rank + 1) * n])
                self.sinks[li, p] = None if a.sink is None else f32([a.sink] * n)
        self.stream_hook = None  # called with (layer, fp32 residual stream) after every specified layer (eager passes only)
        self.scale = 1.0 / math.sqrt(cfg.head_dim)
        if cfg.multi_latent_attention:
            from slime_b200.models import mixers

            self.rope = mixers.mla_rope_table(cfg, max_context + 1, self.device)
            self.scale = mixers.mla_softmax_scale(cfg)
        self.graphs: dict[int, tuple] = {}
        self.replayed_launches = 0  # kernel-library launches executed through graph replays
        self.graph_buckets = [b for b in (1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 192, 256, 384, 512) if b <= max_batch]
        if max_batch not in self.graph_buckets:
            self.graph_buckets.append(max_batch)
        self._static = None
        # expert choices of the tokens of the current forward pass, one [T, k] tensor per MoE layer (routing replay)
        self.record_routed = False
        self._moe_layer_idx = torch.tensor([i for i in range(cfg.num_layers) if cfg.is_moe_layer(i)], dtype=torch.long,
                                           device=self.device)  # fmt: skip
        self._routed: list[torch.Tensor] = []
        self.last_routed = None
        self.last_logits = None  # fp32 logits of the last decode step, one row per slot (a buffer of the graph)
        self.last_hidden = None  # residual stream before the final norm of the last prefill pass, all rows (draft heads read it)

    def take_routed(self):
        """``[T, layers, k]`` int32 expert ids of the pass just run, one column per layer of the model (zeros for dense
        layers: the consumer indexes by layer number); None when not recording."""
        if not self._routed:
            return None
        picked = torch.stack(self._routed, 1)
        self._routed = []
        if self._moe_layer_idx.numel() == self.cfg.num_layers:
            return picked
        out = picked.new_zeros(picked.shape[0], self.cfg.num_layers, picked.shape[2])
        return out.index_copy_(1, self._moe_layer_idx, picked)  # the index lives on the device: capturable

    # ------------------------------------------------------------------ layer math
    def _tp_reduce(self, x):
        if self.tp_group is not None:
            import torch.distributed as dist

            dist.all_reduce(x, group=self.tp_group)
        return x

    def _gather_logits(self, logits):
        """Vocab-parallel LM head: [T, V/tp] per rank -> [T, V] on every rank (rank r owns columns r*V/tp ...)."""
        V = self.cfg.vocab_size  # columns past it are padding of the vocabulary sharding: never sampled, never scored
        if self.tp_group is None or self.w.tp == 1:
            return logits if logits.shape[1] == V else logits[:, :V]
        import torch.distributed as dist

        T, vl = logits.shape
        parts = torch.empty(self.w.tp * T, vl, dtype=logits.dtype, device=logits.device)  # rank-major concatenation
        dist.all_gather_into_tensor(parts, logits.contiguous(), group=self.tp_group)
        full = parts.view(self.w.tp, T, vl).permute(1, 0, 2).reshape(T, -1)
        return full if full.shape[1] == V else full[:, :V]

    def _row_parallel_norm(self, inp, weight, ln, res, T: int, post=None):
        """``rmsnorm(sum over TP ranks of inp @ weight^T + res)`` -> (normed, new residual); ``post``: a sandwich norm
        applied to the projected sum before it joins the residual stream."""
        if post is not None:
            x = self._post_norm(self._tp_reduce(_linear(inp, weight)), post)
            return ops.rmsnorm(x, ln, self.cfg.norm_epsilon, res)
        if self._fused_tp is not None and T <= self._fused_tp.max_tokens:
            _linear(inp, weight, out=self._fused_tp.partial(T))
            return self._fused_tp(T, res, ln, self.cfg.norm_epsilon)
        x = self._tp_reduce(_linear(inp, weight, out_dtype=self._proj_dtype))
        return ops.rmsnorm(x, ln, self.cfg.norm_epsilon, res)

    def _mlp(self, L, x):
        if "gate_up" in L:
            act = ops.swiglu(_linear(x, L["gate_up"]))
            return self._tp_reduce(_linear(act, L["down"], out_dtype=self._proj_dtype))
        return self._moe(L, x)

    def _route(self, L, logits):
        """Expert choice and weights of every token, as the trainer's router computes them."""
        cfg = self.cfg
        from slime_b200.ops import grouped

        if cfg.moe_router_num_groups and cfg.moe_router_group_topk and cfg.moe_router_num_groups > 1:
            return grouped.route_topk(logits, cfg.moe_router_topk, score="sigmoid", renorm=cfg.norm_topk_prob, bias=L.get("router_bias"),
                                      scale=cfg.moe_router_topk_scaling_factor, groups=(cfg.moe_router_num_groups, cfg.moe_router_group_topk))  # fmt: skip
        return grouped.route_topk(logits, cfg.moe_router_topk, score=cfg.moe_router_score_function,
                                  pre_softmax=cfg.moe_router_pre_softmax, renorm=cfg.norm_topk_prob,
                                  bias=L.get("router_bias"), scale=cfg.moe_router_topk_scaling_factor)  # fmt: skip

    def _moe(self, L, x):
        from slime_b200.ops import grouped

        probs, idx = self._route(L, ops.router_gemm(x, L["router"]))
        if self.record_routed:
            self._routed.append(idx.to(torch.int32))
        # expert-sorted, tile-padded layout built on the device (no host sync: the step stays graph-capturable), then
        # one grouped GEMM per projection over all experts

        lay = grouped.DeviceLayout(idx, L["w13"].shape[0], self.w.first_expert)
        y = lay.combine(_grouped_linear(ops.swiglu(_grouped_linear(lay.pad(x), L["w13"], lay)), L["w2"], lay), probs, x.shape[0])
        shared = None
        if "shared_gate_up" in L:  # always-on expert, tensor-parallel like a dense MLP
            shared = _linear(ops.swiglu(_linear(x, L["shared_gate_up"])), L["shared_down"])
            if L.get("shared_gate") is not None:
                shared = shared * torch.sigmoid(x.float() @ L["shared_gate"].float().t()).to(shared.dtype)
        if self.w.ep > 1:  # expert outputs and the shared expert's partial sums travel in one reduction
            return self._tp_reduce(y if shared is None else y + shared)
        if shared is not None:
            y = y + (self._tp_reduce(shared) if self.w.tp > 1 else shared)
        return y

    def _qkv(self, L, normed, positions, slots, li):
        """Packed q / k / v of the new tokens, rotated (and per-head normalised) in place, k and v also written to
        their cache slots of layer ``li``: one GEMM and one fused launch."""
        cfg = self.cfg
        qkv = _linear(normed, L["qkv"], bias=L["qkv_bias"])
        if not self._composed_attention:
            return ops.rope_kv_write(qkv, positions, self.rope, slots, self.kv.k[self.kv_of[li]], self.kv.v[self.kv_of[li]], self.w.hq, self.w.hkv,
                                     cfg.head_dim, L["q_norm"], L["k_norm"], cfg.norm_epsilon)  # fmt: skip
        # attention variants the fused kernel does not cover (partial / interleaved rotary, RMSNorm over all heads):
        # the same steps as separate ops, then the ordinary cache write
        from slime_b200.models import mixers

        T, d, hq, hkv = qkv.shape[0], cfg.head_dim, self.w.hq, self.w.hkv
        q, k, v = qkv.split([hq * d, hkv * d, hkv * d], dim=-1)
        if L["q_norm"] is not None:
            if cfg.qk_layernorm_full:
                q, k = self._full_norm(q, L["q_norm"]), self._full_norm(k, L["k_norm"])
            else:
                q = mixers._rms(q.view(T, hq, d), L["q_norm"], cfg.norm_epsilon).view(T, -1)
                k = mixers._rms(k.view(T, hkv, d), L["k_norm"], cfg.norm_epsilon).view(T, -1)
        if self.rope.shape[1] > 0:
            cos, sin = mixers.rotary_cos_sin(self.rope, positions, self._band_axes() if positions.dim() == 2 else None)
            q = mixers.apply_rotary(q.view(T, hq, d), cos, sin, cfg.rotary_interleaved).view(T, -1)
            k = mixers.apply_rotary(k.view(T, hkv, d), cos, sin, cfg.rotary_interleaved).view(T, -1)
        k, v = k.contiguous(), v.contiguous()
        ops.kv_write(k, v, slots, self.kv.k[self.kv_of[li]], self.kv.v[self.kv_of[li]])
        return torch.cat([q, k, v], dim=-1)

    def _band_axes(self):
        if self._mrope_axes is None:
            from slime_b200.models.vision import mrope_band_axes

            self._mrope_axes = mrope_band_axes(self.cfg.mrope_section, self.rope.shape[1] // 2, self.cfg.mrope_interleaved, self.device)
        return self._mrope_axes

    @torch.no_grad()
    def encode_images(self, pixel_values, grid_thw):
        """Image encoder outputs [placeholder tokens, H] for one request's images, and the list of same-shaped vectors
        that join the stream after the first layers (empty unless the encoder has deepstack outputs)."""
        out, extras = self.w.vision(pixel_values.to(self.device), grid_thw.to(self.device), with_deepstack=True)
        return out.to(self.w.dtype), [e.to(self.w.dtype) for e in extras]

    def _full_norm(self, t, w):
        """RMSNorm over all heads of the model: the sum of squares crosses the tensor-parallel ranks."""
        f = t.float()
        ss = f.pow(2).sum(-1, keepdim=True)
        n = f.shape[-1] * self.w.tp
        if self.w.tp > 1:
            ss = self._tp_reduce(ss)
        return (f * torch.rsqrt(ss / n + self.cfg.norm_epsilon) * w.float()).to(t.dtype)

    # ------------------------------------------------------------ latent attention layers
    def _mla_project(self, L, x, positions, slots, li):
        """Queries [T, hq, dn + dr] (rotary part rotated) of the new tokens; their latent vectors (normalised compressed
        key/value + rotated shared key) are written to the cache slab of layer ``li`` and returned [T, kv_lora + dr]."""
        from slime_b200.models import mixers

        cfg, T = self.cfg, x.shape[0]
        dn, dr = cfg.qk_head_dim, cfg.qk_pos_emb_head_dim
        hq = cfg.num_attention_heads // self.w.tp
        if "q_a" in L:
            q = ops.gemm(mixers._rms(ops.gemm(x, L["q_a"]), L["q_a_ln"], cfg.norm_epsilon), L["q_b"])
        else:
            q = ops.gemm(x, L["q_proj"])
        q = q.view(T, hq, dn + dr)
        c_kv, k_pe = ops.gemm(x, L["kv_a"]).split([cfg.kv_lora_rank, dr], dim=-1)
        cos, sin = mixers.rotary_cos_sin(self.rope, positions)
        q = torch.cat([q[..., :dn], mixers.apply_rotary(q[..., dn:], cos, sin, cfg.rotary_interleaved)], dim=-1)
        k_pe = mixers.apply_rotary(k_pe.reshape(T, 1, dr), cos, sin, cfg.rotary_interleaved).reshape(T, dr)
        parts = [mixers._rms(c_kv, L["kv_a_ln"], cfg.norm_epsilon), k_pe]
        index_q = None
        if cfg.index_topk:  # every layer caches an indexer key slot (unused on layers that reuse another layer's choice)
            hi, di = cfg.index_n_heads, cfg.index_head_dim
            if "idx_wk" in L:
                q_latent = mixers._rms(ops.gemm(x, L["q_a"]), L["q_a_ln"], cfg.norm_epsilon)
                il = cfg.rotary_interleaved if cfg.index_rotary_interleaved is None else cfg.index_rotary_interleaved
                qi = mixers.apply_rotary(ops.gemm(q_latent, L["idx_wq_b"]).view(T, hi, di), cos, sin, il)
                ki = torch.nn.functional.layer_norm(ops.gemm(x, L["idx_wk"]).float(), (di,), L["idx_k_norm_w"].float(), L["idx_k_norm_b"].float())
                ki = mixers.apply_rotary(ki.view(T, 1, di), cos, sin, il).view(T, di)
                wi = ops.gemm(x, L["idx_weights"]).float() * (hi**-0.5) * (di**-0.5)
                index_q = (qi.float(), wi)
                parts.append(ki.to(x.dtype))
            else:
                parts.append(x.new_zeros(T, di))
        latent = torch.cat(parts, dim=-1).contiguous()
        cache = self.kv.k[self.kv_of[li]]
        ok = slots >= 0
        cache.view(cache.shape[0], -1)[slots[ok].long()] = latent[ok].to(cache.dtype)
        return q, latent, index_q

    def _dsa_restrict(self, L, li, index_q, lat, allowed):
        """Keep, per query row, the ``index_topk`` cached tokens the indexer scores highest (rows that see fewer keep all).
        The choice is remembered for the layers of this pass that reuse it."""
        cfg = self.cfg
        if not cfg.index_topk:
            return allowed
        if index_q is None:
            return self._dsa_masks[L["index_source"]]
        if allowed.shape[1] > cfg.index_topk:
            qi, wi = index_q
            ki = lat[..., cfg.kv_lora_rank + cfg.qk_pos_emb_head_dim :].float()
            logits = (torch.einsum("bhd,bld->bhl", qi, ki).relu_() * wi[:, :, None]).sum(1).masked_fill(~allowed, float("-inf"))
            pick = torch.zeros_like(allowed).scatter_(1, logits.topk(cfg.index_topk, dim=-1).indices, True)
            allowed = pick & allowed
        self._dsa_masks[li] = allowed
        return allowed

    def _mla_absorbed(self, L, q, latent, allowed):
        """Attention of queries ``q`` [B, hq, dn + dr] over per-row latent contexts ``latent`` [B, Lmax, kv_lora + dr] with
        ``allowed`` [B, Lmax]: the key expansion is folded into the query and the value expansion applied after the
        weighted sum, so the cached vector is never expanded per head. Returns [B, hq * dv]."""
        cfg = self.cfg
        dn, dv, r = cfg.qk_head_dim, cfg.v_head_dim, cfg.kv_lora_rank
        hq = q.shape[1]
        dr = cfg.qk_pos_emb_head_dim
        w = L["kv_b"].float().view(hq, dn + dv, r)
        q_lat = torch.einsum("bhd,hdr->bhr", q[..., :dn].float(), w[:, :dn])  # queries in latent coordinates
        lat = latent.float()
        scores = (torch.einsum("bhr,blr->bhl", q_lat, lat[..., :r]) + torch.einsum("bhd,bld->bhl", q[..., dn:].float(), lat[..., r : r + dr]))
        scores = (scores * self.scale).masked_fill(~allowed[:, None, :], float("-inf"))
        out_lat = torch.einsum("bhl,blr->bhr", scores.softmax(-1), lat[..., :r])
        return torch.einsum("bhr,hdr->bhd", out_lat, w[:, dn:]).reshape(q.shape[0], hq * dv).to(self.w.dtype)

    def _mla_prefill(self, L, li, x, positions, slots, cu_q, kv_gather_slots, cu_k, fresh):
        q, latent, index_q = self._mla_project(L, x, positions, slots, li)
        cache = self.kv.k[self.kv_of[li]]
        ctx_lat = latent if fresh else cache.view(cache.shape[0], -1).index_select(0, kv_gather_slots)
        cq, ck = cu_q.tolist(), (cu_q if fresh else cu_k).tolist()
        lmax = max(b - a for a, b in zip(ck[:-1], ck[1:]))
        T = x.shape[0]
        lat = ctx_lat.new_zeros(T, lmax, ctx_lat.shape[-1])
        allowed = torch.zeros(T, lmax, dtype=torch.bool, device=x.device)
        for (qa, qb), (ka, kb) in zip(zip(cq[:-1], cq[1:]), zip(ck[:-1], ck[1:])):
            n_q, n_k = qb - qa, kb - ka
            if n_q <= 0:
                continue
            lat[qa:qb, :n_k] = ctx_lat[ka:kb]
            allowed[qa:qb, :n_k] = torch.ones(n_q, n_k, dtype=torch.bool, device=x.device).tril(diagonal=n_k - n_q)
        return self._mla_absorbed(L, q, lat, self._dsa_restrict(L, li, index_q, lat, allowed))

    def _mla_decode(self, L, li, x, positions, slots, block_table, seq_lens, n):
        q, _, index_q = self._mla_project(L, x, positions, slots, li)
        cache = self.kv.k[self.kv_of[li]]
        ps = self.kv.page_size
        lmax = int(seq_lens.max())
        pos = torch.arange(lmax, device=x.device)
        idx = block_table[:, (pos // ps).clamp_max(block_table.shape[1] - 1)].long() * ps + pos % ps  # [n, lmax]
        lat = cache.view(cache.shape[0], -1)[idx.clamp_(0, cache.shape[0] - 1)]
        return self._mla_absorbed(L, q, lat, self._dsa_restrict(L, li, index_q, lat, pos[None, :] < seq_lens[:, None]))

    # ------------------------------------------------------------ gated delta-net layers
    def _gdn_project(self, L, x):
        """Input projections of a delta-net layer -> (pre-convolution q|k|v channels [T, C], z [T, Hv, Dv], b, a [T, Hv])."""
        cfg, T = self.cfg, x.shape[0]
        hk, hv, dk, dv = cfg.linear_num_key_heads, cfg.linear_num_value_heads, cfg.linear_key_head_dim, cfg.linear_value_head_dim
        if "gdn_qkvz" in L:  # rows grouped per key head: q, k, then that head's value and gate heads
            r = hv // hk
            qkvz = ops.gemm(x, L["gdn_qkvz"]).view(T, hk, 2 * dk + 2 * r * dv)
            q, k, v, z = qkvz.split([dk, dk, r * dv, r * dv], dim=-1)
            b, a = ops.gemm(x, L["gdn_ba"]).view(T, hk, 2 * r).split([r, r], dim=-1)
            mixed = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=-1)
            return mixed, z.reshape(T, hv, dv), b.reshape(T, hv), a.reshape(T, hv)
        return ops.gemm(x, L["gdn_qkv"]), ops.gemm(x, L["gdn_z"]).view(T, hv, dv), ops.gemm(x, L["gdn_b"]), ops.gemm(x, L["gdn_a"])

    def _gdn(self, L, li, x, recur):
        """Delta-net layer; ``recur`` as in ``_specified_layers``."""
        cfg, T = self.cfg, x.shape[0]
        hk, hv, dk, dv = cfg.linear_num_key_heads, cfg.linear_num_value_heads, cfg.linear_key_head_dim, cfg.linear_value_head_dim
        mixed, z, b, a = self._gdn_project(L, x)
        q, k, v = mixed.contiguous().split([hk * dk, hk * dk, hv * dv], dim=-1)
        inputs = delta.DeltaInputs(q, k, v, a, b, L["gdn_conv"], L["gdn_A_log"], L["gdn_dt_bias"])
        return ops.gemm(recur(self.state_of[li], inputs.gated(z.reshape(T, -1), L["gdn_norm"], "silu", cfg.norm_epsilon), None), L["gdn_out"])

    def _extend_recurrence(self, extend):
        """``recur(state number, mixer, output view or None)`` of an extend pass; ``mixer``: ``ops.delta.DeltaMixer`` or one of
        ``ops.linear_scan``."""
        return lambda n, mixer, out: mixer.extend(self.states.of[n], extend, out)

    def _step_recurrence(self, n_rows: int, positions):
        """The same of a decode step: idle rows touch no state."""
        slots, active = self._static["state_slot"][:n_rows], self._static["active"][:n_rows]
        return lambda n, mixer, out: mixer.step(self.states.of[n], slots, active, positions, out)

    # ------------------------------------------------------------ specified layers (models/layer_spec.py)
    def _specified_layers(self, ids, prev, positions, slots, attend, attend_latent, recur):
        """All layers of a model with ``layer_specs`` over the tokens ``ids`` (``prev``: the tokens in front of them, -1 at a
        sequence's start; read by models with a bigram table) -> the final norm's output. ``attend(slab, spec, q, form, out)`` runs an
        attention mixer once the keys and values of cache slab ``slab`` are there, ``attend_latent(slab, latent, q, gate, out)`` a latent one,
        ``recur`` (``_extend_recurrence``) a recurrent one: the
        only parts that differ between a prefill pass and a decode step. The residual stream is fp32; between two
        sub-layers there is one fused launch (which hands on the stream itself where a model has no norms of inputs)."""
        cfg, w = self.cfg, self.w
        norm = dict(kind=cfg.norm_kind, offset=cfg.norm_offset, groups=cfg.norm_groups, emit=w.dtype)
        f32, eps = torch.float32, cfg.norm_epsilon
        first = w.layers[0].get("ln1")
        pair = None
        if cfg.bigram:
            pair = stream.PairTable(w.bigram, ids.to(torch.int32), prev, cfg.bigram["mul_prev"], cfg.bigram["mul_cur"])
        if w.tp > 1:  # vocab-parallel table: rows of other ranks come out as zeros
            x = self._tp_reduce(stream.stream_norm(w.embed, None, None, eps, ids=ids - w.rank * w.vocab_local)[1])
            if pair is not None:
                x = x + pair.table[pair.rows()].float()
            h, res = stream.stream_norm(x, None, first, eps, post_w=w.embed_norm, **norm)
        else:
            h, res = stream.stream_norm(w.embed, None, first, eps, ids=ids, pair=pair, post_w=w.embed_norm, **norm)
        for li, L in enumerate(w.layers):
            spec, last = L["spec"], li + 1 == len(w.layers)
            after, gain = (w.final_norm, cfg.logit_scale) if last else (w.layers[li + 1].get("ln1"), 1.0)
            behind = spec.mlp is not None and not spec.parallel_ff
            y = _linear(self._specified_mixers(L, li, h, positions, slots, attend, attend_latent, recur), L["out"], bias=L.get("out_bias"), out_dtype=f32)
            if spec.parallel_ff and spec.mlp is not None and spec.mlp.experts is not None:
                y = self._specified_experts(L, spec.mlp, h, y)
            else:
                y = self._tp_reduce(y)
            h, _ = stream.stream_norm(y, res, L.get("ln2") if behind else after, eps, post_w=L.get("post_attn_ln"), gain=1.0 if behind else gain, **norm)
            if behind:
                h, _ = stream.stream_norm(self._specified_mlp(L, spec.mlp, h), res, after, eps, post_w=L.get("post_mlp_ln"), gain=gain, **norm)
            if self.stream_hook is not None:
                self.stream_hook(li, res)
        return h

    def _specified_mixers(self, L, li, h, positions, slots, attend, attend_latent, recur):
        """What goes into a layer's output projection: the heads of its mixers, scaled, and the hidden units of a feed-forward
        beside them, side by side as in ``LayerProjections.outs``."""
        spec, lay, T = L["spec"], L["proj"], h.shape[0]
        x = _linear(h, L["in"], bias=L.get("in_bias"))
        cols = lambda name: x[:, lay.ins[name][0] : sum(lay.ins[name])]  # noqa: E731
        y = (torch.zeros if lay.padded(lay.outs) else torch.empty)(T, lay.out_cols, dtype=h.dtype, device=h.device)
        slab, number, eps = self.kv_of[li], self.state_of[li], self.cfg.norm_epsilon
        for p, m, factor in spec.branches():
            c0, n = lay.outs[p + "o"]
            out = y[:, c0 : c0 + n]
            if isinstance(m, AttentionSpec):
                own = m.kv_from is None
                at = slab if own else self.kv_of[m.kv_from]  # where its keys and values are
                slab = slab + 1 if own else slab
                q, k, v, sums = cols(p + "q"), None, None, None
                if own:
                    k = cols(p + "k")
                    v = k if m.tied_values else cols(p + "v")
                if m.qk_norm and m.norm_over == "projection" and self.w.tp > 1:
                    sums = (self._tp_reduce(stream.head_sums(q, k)), m.norm_widths())
                q = stream.place_heads(q, k, v, slots, self.kv.k[at], self.kv.v[at], q_norm=L.get(p + "q.norm"), k_norm=L.get(p + "k.norm"),
                                       eps=eps, table=self.rotary.get(m.rot), positions=positions, interleaved=m.rot is None or m.rot.interleaved,
                                       sums=sums, maps=m.maps)  # fmt: skip
                form = dict(slopes=self.slopes[li, p], sinks=self.sinks[li, p], out_scale=factor, chunk=m.chunk, softcap=m.softcap,
                            bias=L.get(p + "bias"), gate=cols(p + "g") if m.gate else None)  # fmt: skip
                if m.diff is not None:
                    form["pair"] = window_attention.Pair(L[p + "pair"], factor * (1.0 - m.diff), eps)
                attend(at, m, q, form, out)
                continue
            if isinstance(m, LatentSpec):
                heads, table = m.heads // self.w.tp, self.rotary[m.rot]
                c = latent.latent_place(cols(p + "dq"), cols(p + "dkv"), L[p + "dq.norm"], L[p + "dkv.norm"], eps, table,
                                        positions, slots, self.kv.k[slab], m.rot.interleaved)  # fmt: skip
                q = _linear(c, L[p + "up_q"]).view(T, heads, m.dim + m.rot_dim)
                gate = cols(p + "g").unflatten(1, (heads, m.vdim)) if m.gate else None
                sizes = latent.Latent(heads, m.dim, m.vdim, m.kv_rank, m.scale, L[p + "up_q"], L[p + "up_kv"], table, m.rot.interleaved)
                attend_latent(slab, sizes, q, gate, out.unflatten(1, (heads, m.vdim)))
                if factor != 1.0:
                    out.mul_(factor)
                slab += 1
                continue
            if isinstance(m, StateSpaceSpec):
                mixer = linear_scan.StateSpace(*(cols(p + n) for n in ("z", "x", "B", "C", "dt")), L[p + "conv"], L[p + "conv.b"], L[p + "A_log"],
                                               L[p + "dt_bias"], L[p + "D"], L[p + "norm"], m.norm_groups // self.w.tp, eps, factor)  # fmt: skip
                recur(number, mixer, out)
                number += 1
                continue
            if isinstance(m, MatrixMemorySpec):
                recur(number, linear_scan.MatrixMemory(*(cols(p + n) for n in "qkvifg"), L[p + "i.b"], L[p + "f.b"], L[p + "norm"], m.gate_cap, eps,
                                                       factor), out)  # fmt: skip
                number += 1
                continue
            a, z = (cols(p + s) if p + s in lay.ins else None for s in "ag")
            if p in lay.low:
                r0, inner, _, parts = lay.low[p]
                second = _linear(x[:, r0 : r0 + inner], L[p + "low"])
                if p + "a2" in parts:
                    a = second[:, parts[p + "a2"][0] : sum(parts[p + "a2"][:2])]
                if p + "g2" in parts:
                    z = second[:, parts[p + "g2"][0] : sum(parts[p + "g2"][:2])]
            inputs = delta.DeltaInputs(cols(p + "q"), cols(p + "k"), cols(p + "v"), a, cols(p + "b"), L[p + "conv"], L[p + "A_log"], L[p + "dt_bias"])
            recur(number, inputs.gated(z, L[p + "norm"], m.gate, eps, factor), out)
            number += 1
        if lay.ff is not None:
            m, (c0, n), r0 = spec.mlp, lay.outs[spec.joint_ff[0] + ".down"], lay.ff[0]
            stream.feed_forward_act(x[:, r0 : r0 + (2 * n if m.gated else n)], m.act, m.gated, out=y[:, c0 : c0 + n])
        return y

    def _specified_mlp(self, L, m, h):
        """Feed-forward behind the mixer of a specified layer: fp32 output, or for experts the unfinished sum the next norm completes."""
        w, f32 = self.w, torch.float32
        if m.experts is None:
            act = _linear(h, L["gate_up"])
            if m.act == "poly_norm":
                sums = self._tp_reduce(stream.poly_sums(act)) if w.tp > 1 else None
                act = stream.poly_norm(act, L["act_coef"], self.cfg.norm_epsilon, sums, m.ff)
            else:
                act = stream.feed_forward_act(act, m.act, m.gated)
            return self._tp_reduce(_linear(act, L["down"], out_dtype=f32))
        out = self._expert_rows(L, m, h)
        if m.shared_ff:
            out.shared = _linear(stream.feed_forward_act(_linear(h, L["shared_gate_up"]), m.act, m.gated), L["shared_down"])
        if w.ep > 1:  # this rank's experts and its part of the shared one travel in one reduction
            return self._tp_reduce(stream.combine(out))
        if w.tp > 1 and out.shared is not None:
            out.shared = self._tp_reduce(out.shared)
        return out

    def _specified_experts(self, L, m, h, y):
        """Experts beside a mixer: the unfinished sum of both, ``y`` being this rank's part of the mixer's output (and of the shared
        expert's)."""
        out = self._expert_rows(L, m, h)
        out.base = y if self.w.ep > 1 else self._tp_reduce(y)
        return self._tp_reduce(stream.combine(out)) if self.w.ep > 1 else out

    def _expert_rows(self, L, m, h) -> stream.ExpertSum:
        """Routing and the experts' products."""
        f32 = torch.float32
        from slime_b200.ops import grouped

        # bf16 products are exact in fp32, so the tensor-core product is a 32-bit router too; the CUDA-core kernel is the
        # faster one for a handful of tokens
        big = h.is_cuda and h.dtype == torch.bfloat16 and h.shape[0] >= 256
        logits = ops.gemm(h, L["router"], out_dtype=f32, splitk=1) if big else ops.router_gemm(h, L["router"])
        probs, idx = grouped.route_topk(logits[:, : m.experts], m.top, score=m.score, renorm=m.renorm, raw_index=True, shift=L.get("router_shift"),
                                        groups=(m.expert_groups, m.keep_groups))  # fmt: skip
        if self.record_routed:
            pad = self.cfg.moe_router_topk - m.top
            self._routed.append(torch.nn.functional.pad(idx.to(torch.int32), (0, pad)) if pad else idx.to(torch.int32))
        lay = grouped.DeviceLayout(idx, L["w13"].shape[0], L["first_expert"])
        rows = _grouped_linear(stream.feed_forward_act(_grouped_linear(lay.pad(h), L["w13"], lay), m.act, m.gated), L["w2"], lay)
        return stream.ExpertSum(rows, lay.slot_dest, probs, gate=logits[:, m.experts] if m.shared_gate else None)

    def _post_norm(self, x, w):
        """GLM-4 sandwich norm: the sub-layer's output is normalised before it joins the residual stream."""
        return x if w is None else ops.rmsnorm(x, w, self.cfg.norm_epsilon)[0]

    # --------------------------------------------------------------------- prefill
    @torch.no_grad()
    def prefill(self, ids, positions, slots, cu_q, kv_gather_slots, cu_k, max_q, max_k, last_rows, fresh: bool, prev=None,
                embed_rows=None, extend=None):
        """Extend pass over packed new tokens.

        ids/positions/slots: [T] for the new tokens; ``cu_q`` their per-request boundaries.
        ``kv_gather_slots``/``cu_k``: cache slots of every context token (cached prefix + new) per
        request, used when some context is already cached (``fresh`` False). Returns logits
        ``[len(last_rows), V/tp]`` fp32 for the requested rows and, when ``last_rows`` is None, all rows.
        ``prev``: the token in front of each row (-1 at a sequence's start), for models with a bigram table.
        Vision inputs: ``positions`` may be ``[3, T]`` (temporal / height / width streams) and ``embed_rows`` = (rows,
        vectors) replaces the embeddings of image placeholder tokens by the encoder's outputs.
        Models with specified layers read the context from the cache pages, models with recurrent mixers continue each
        request's state: ``extend`` (``ops.window_attention.ExtendBatch``) says where every row stands. With specified layers
        ``kv_gather_slots`` is not used.
        """
        cfg, w, d = self.cfg, self.w, self.cfg.head_dim
        if self.layered:
            def attend(n, a, q, form, out):
                return window_attention.window_extend(q, self.kv.k[n], self.kv.v[n], extend, a.scale, a.window, a.keep_first, out=out, **form)

            def attend_latent(n, sizes, q, gate, out):
                return latent.latent_extend(sizes, q, self.kv.k[n], extend, gate, out)

            h = self._specified_layers(ids, prev, positions, slots, attend, attend_latent, self._extend_recurrence(extend))
            h = h if last_rows is None else h.index_select(0, last_rows)
            return self.logits_of(h)
        x = ops.embedding(ids, w.embed, w.rank * w.vocab_local)
        x = self._tp_reduce(x) if w.tp > 1 else x
        deepstack = []
        if embed_rows is not None:
            x = x.index_copy(0, embed_rows[0], embed_rows[1].to(x.dtype))
            deepstack = embed_rows[2] if len(embed_rows) > 2 else []
        res = None
        T = ids.numel()
        recur = self._extend_recurrence(extend)
        for li, L in enumerate(w.layers):
            if 0 < li <= len(deepstack):  # vision vectors that join the stream after layer li - 1 (stream = x + res)
                x = x.index_add(0, embed_rows[0], deepstack[li - 1].to(x.dtype))
            normed, res = ops.rmsnorm(x, L["ln1"], cfg.norm_epsilon, res)
            if L["kind"] == "gdn":
                x = self._gdn(L, li, normed, recur)
                normed, res = ops.rmsnorm(x, L["ln2"], cfg.norm_epsilon, res)
                x = self._mlp(L, normed)
                continue
            if L["kind"] == "mla":
                ctx = self._mla_prefill(L, li, normed, positions, slots, cu_q, kv_gather_slots, cu_k, fresh)
                x = self._tp_reduce(_linear(ctx, L["o"], out_dtype=self._proj_dtype))
                normed, res = ops.rmsnorm(x, L["ln2"], cfg.norm_epsilon, res)
                x = self._mlp(L, normed)
                continue
            qkv = self._qkv(L, normed, positions, slots, li)
            q3 = qkv.view(T, w.hq + 2 * w.hkv, d)
            q, k, v = q3[:, : w.hq], q3[:, w.hq : w.hq + w.hkv], q3[:, w.hq + w.hkv :]
            if fresh:
                ctx = ops.varlen_attention(q, k, v, cu_q, max_q, self.scale, sinks=L.get("sinks"))
            else:
                k_all = self.kv.k[self.kv_of[li]].index_select(0, kv_gather_slots)
                v_all = self.kv.v[self.kv_of[li]].index_select(0, kv_gather_slots)
                ctx = _extend_attention(q, k_all, v_all, cu_q, cu_k, max_q, max_k, self.scale, sinks=L.get("sinks"))
            ctx = ctx.reshape(T, -1)
            if "gate" in L:
                ctx = ctx * torch.sigmoid(ops.gemm(normed, L["gate"]).float()).to(ctx.dtype)
            x = self._tp_reduce(_linear(ctx, L["o"], out_dtype=self._proj_dtype))
            x = self._post_norm(x, L["post_attn_ln"])
            normed, res = ops.rmsnorm(x, L["ln2"], cfg.norm_epsilon, res)
            x = self._post_norm(self._mlp(L, normed), L["post_mlp_ln"])
        h, hidden = ops.rmsnorm(x, w.final_norm, cfg.norm_epsilon, res)
        self.last_hidden = hidden if w.draft else None  # kept for a draft head only: a chunk's stream is tens of megabytes
        if last_rows is not None:
            h = h.index_select(0, last_rows)
        return self._gather_logits(ops.gemm(h, w.lm_head, out_dtype=torch.float32))

    @torch.no_grad()
    def draft_extend(self, depth: int, hidden, next_ids, positions, slots, cu_q, kv_gather_slots, cu_k, max_q, max_k, fresh: bool):
        """Draft head ``depth`` over packed rows: row p joins the residual stream ``hidden[p]`` the trunk (or the previous
        draft step) left at position p with the embedding of the token at position p + 1, runs one transformer layer with
        its own cache slab (written at ``slots``) and returns ``(normed [T, H], stream [T, H])``: the first feeds the shared
        output head (a guess for the token at position p + 2), the second is the next draft step's ``hidden``. Same
        computation as ``models/gpt.py::MTPLayer``; arguments as in ``prefill``."""
        cfg, w, d, eps = self.cfg, self.w, self.cfg.head_dim, self.cfg.norm_epsilon
        L, li = w.draft[depth], cfg.num_layers + depth
        recording, self.record_routed = self.record_routed, False  # a draft head's routing is nobody's training signal
        try:
            emb = ops.embedding(next_ids, w.embed, w.rank * w.vocab_local)
            emb = self._tp_reduce(emb) if w.tp > 1 else emb
            e_n = ops.rmsnorm(emb, L["enorm"], eps)[0]
            h_n = ops.rmsnorm(hidden.to(emb.dtype), L["hnorm"], eps)[0]
            x = ops.gemm(torch.cat([e_n, h_n], dim=-1), L["eh_proj"])
            T = x.shape[0]
            normed, res = ops.rmsnorm(x, L["ln1"], eps, None)
            if L["kind"] == "mla":
                ctx = self._mla_prefill(L, li, normed, positions, slots, cu_q, kv_gather_slots, cu_k, fresh)
                x = self._tp_reduce(_linear(ctx, L["o"], out_dtype=self._proj_dtype))
            else:
                qkv = self._qkv(L, normed, positions, slots, li)
                q3 = qkv.view(T, w.hq + 2 * w.hkv, d)
                q, k, v = q3[:, : w.hq], q3[:, w.hq : w.hq + w.hkv], q3[:, w.hq + w.hkv :]
                if fresh:
                    ctx = ops.varlen_attention(q, k, v, cu_q, max_q, self.scale, sinks=L.get("sinks"))
                else:
                    k_all = self.kv.k[self.kv_of[li]].index_select(0, kv_gather_slots)
                    v_all = self.kv.v[self.kv_of[li]].index_select(0, kv_gather_slots)
                    ctx = _extend_attention(q, k_all, v_all, cu_q, cu_k, max_q, max_k, self.scale, sinks=L.get("sinks"))
                ctx = ctx.reshape(T, -1)
                if "gate" in L:
                    ctx = ctx * torch.sigmoid(ops.gemm(normed, L["gate"]).float()).to(ctx.dtype)
                x = self._post_norm(self._tp_reduce(_linear(ctx, L["o"], out_dtype=self._proj_dtype)), L["post_attn_ln"])
            normed, res = ops.rmsnorm(x, L["ln2"], eps, res)
            x = self._post_norm(self._mlp(L, normed), L["post_mlp_ln"])
            return ops.rmsnorm(x, L["final_ln"], eps, res)
        finally:
            self.record_routed = recording

    def logits_of(self, normed):
        """Output head over already normalised rows -> fp32 logits over the whole vocabulary."""
        logits = ops.gemm(normed, self.w.lm_head, out_dtype=torch.float32)
        return self._gather_logits(stream.softcap_(logits, self.cfg.logit_softcap) if self.cfg.logit_softcap else logits)

    # ---------------------------------------------------------------------- decode
    # Per-slot decode state is device-owned (ids / pos / out_pos): the token sampled in step t is the
    # input of step t+1 without touching the host, so steps can be launched back to back while the host
    # lags one step behind reading results. The host owns the block table, the active mask, sampling
    # parameters and "init" records for slots that start decoding; those live in one flat pinned buffer
    # (double-buffered) uploaded with a single copy per step.
    HOST_FIELDS = ("active", "init_mask", "init_ids", "init_pos", "init_out_pos", "init_prev", "state_slot", "top_k", "temperature", "top_p", "min_p")

    def _alloc_static(self):
        B, W, dev = self.max_batch, self.max_pages_per_req, self.device
        nf = len(self.HOST_FIELDS)
        total = (nf + 2) * B + B * W
        self._flat_dev = torch.zeros(total, dtype=torch.int32, device=dev)
        self._flat_hosts = [torch.zeros(total, dtype=torch.int32, pin_memory=(dev.type == "cuda")) for _ in range(2)]
        self._host_events = [None, None]
        self._host_idx = 0

        def views(flat):
            out, off = {"seeds": flat[: 2 * B].view(torch.int64)}, 2 * B  # 8-byte fields first: any number of slots is fine
            for f in self.HOST_FIELDS:
                v = flat[off : off + B]
                out[f] = v.view(torch.float32) if f in ("temperature", "top_p", "min_p") else v
                off += B
            out["block_table"] = flat[off : off + B * W].view(B, W)
            return out

        self._static = views(self._flat_dev)
        # the scheduler edits `host` (plain numpy, not pinned); upload copies it into the free pinned buffer
        import numpy as np

        self._host_np = np.zeros(total, dtype=np.int32)
        self.host = {k: v.numpy() for k, v in views(torch.from_numpy(self._host_np)).items()}
        self.host["temperature"][:] = 1.0
        self.host["top_p"][:] = 1.0
        i32 = lambda *sh: torch.zeros(*sh, dtype=torch.int32, device=dev)  # noqa: E731
        self._dev_state = dict(ids=i32(B), pos=i32(B), out_pos=i32(B), ids_eff=i32(B), pos_eff=i32(B), seq_lens=i32(B) + 1,
                               slots=i32(B))  # fmt: skip
        if self.cfg.bigram:  # the token in front of each slot's current one
            self._dev_state.update(prev=i32(B) - 1, prev_eff=i32(B) - 1)

    def upload_static(self):
        """Copy the scheduler's host state to the device through a pinned staging buffer that is not in
        flight (two alternate; an event guards reuse). ``init_mask`` is consumed by the upload."""
        k = self._host_idx
        ev = self._host_events[k]
        if ev is not None:
            ev.synchronize()
        stage = self._flat_hosts[k]
        stage.numpy()[:] = self._host_np
        self._flat_dev.copy_(stage, non_blocking=True)
        if self.device.type == "cuda":
            ev = torch.cuda.Event()
            ev.record()
            self._host_events[k] = ev
        self._host_idx = 1 - k
        self.host["init_mask"][:] = 0
        return stage.numel() * 4

    def _decode_step(self, n: int, filtered: bool, kept_cap: int):
        """prepare -> model -> sample -> advance for slots [0, n). Returns (tokens, logprobs, kept_ids, kept_cnt, routed
        experts, logits)."""
        w = self.w
        st, ds = self._static, self._dev_state
        ps, W = self.kv.page_size, self.max_pages_per_req
        ids, pos, seq_lens, slots = ds["ids_eff"][:n], ds["pos_eff"][:n], ds["seq_lens"][:n], ds["slots"][:n]
        bt = st["block_table"][:n]
        if self.device.type == "cuda":
            from slime_b200.ops import _lib

            P = _lib.ptr
            _lib.check(_lib.lib().sb_decode_prepare(
                P(ds["ids"]), P(ds["pos"]), P(ds["out_pos"]), P(st["init_mask"]), P(st["init_ids"]), P(st["init_pos"]),
                P(st["init_out_pos"]), P(st["active"]), P(st["block_table"]), P(ds["ids_eff"]), P(ds["pos_eff"]),
                P(ds["seq_lens"]), P(ds["slots"]), P(ds.get("prev")), P(st["init_prev"]), P(ds.get("prev_eff")), n, ps, W, _lib.stream()), "sb_decode_prepare")  # fmt: skip
        else:
            self._prepare_reference(n)
        h = self._decode_layers(n, ids, pos, slots, bt, seq_lens)
        logits = self.logits_of(h)
        tok, lp, kept_ids, kept_cnt = ops.sample(
            logits, st["temperature"][:n], st["top_k"][:n] if filtered else None, st["top_p"][:n] if filtered else None,
            st["min_p"][:n] if filtered else None, st["seeds"][:n], ds["out_pos"][:n], kept_cap,
        )  # fmt: skip
        routed = self.take_routed()
        if self.device.type == "cuda":
            _lib.check(_lib.lib().sb_decode_advance(P(ds["ids"]), P(ds["pos"]), P(ds["out_pos"]), P(st["active"]), P(tok),
                                                    P(ds.get("prev")), n, _lib.stream()), "sb_decode_advance")  # fmt: skip
        else:
            act = st["active"][:n].bool()
            if "prev" in ds:
                ds["prev"][:n] = torch.where(act, ds["ids"][:n], ds["prev"][:n])
            ds["ids"][:n] = torch.where(act, tok, ds["ids"][:n])
            ds["pos"][:n] += act.int()
            ds["out_pos"][:n] += act.int()
        return tok, lp, kept_ids, kept_cnt, routed, logits

    def _decode_layers(self, n, ids, pos, slots, bt, seq_lens):
        """Embedding to final norm for one token per slot."""
        cfg, w, d, ps = self.cfg, self.w, self.cfg.head_dim, self.kv.page_size
        if self.layered:
            def attend(i, a, q, form, out):
                return window_attention.window_decode(q, self.kv.k[i], self.kv.v[i], bt, seq_lens, pos, ps, a.scale, a.window, a.keep_first,
                                                      max_context=self.max_context, out=out, **form)  # fmt: skip

            def attend_latent(i, sizes, q, gate, out):
                return latent.latent_decode(sizes, q, self.kv.k[i], bt, pos, ps, self.max_context, gate, out)

            prev = self._dev_state["prev_eff"][:n] if cfg.bigram else None
            return self._specified_layers(ids, prev, pos, slots, attend, attend_latent, self._step_recurrence(n, pos))
        recur = self._step_recurrence(n, pos)  # (a state's position counts tokens, whatever the rotary position is)
        if self.rope_delta is not None:
            pos = pos + self.rope_delta[:n]  # rotary position of a request that carries images
        x = ops.embedding(ids, w.embed, w.rank * w.vocab_local)
        x = self._tp_reduce(x) if w.tp > 1 else x
        if self._fused_tp is not None:
            # after the NCCL all-reduce of the vocab-parallel embedding: that collective has already lined the ranks
            # up, so the bounded barrier only ever waits for launch jitter
            self._fused_tp.begin_forward()
        normed, res = ops.rmsnorm(x, w.layers[0]["ln1"], cfg.norm_epsilon, None)
        for li, L in enumerate(w.layers):
            if L["kind"] == "gdn":
                normed, res = ops.rmsnorm(self._gdn(L, li, normed, recur), L["ln2"], cfg.norm_epsilon, res)
            elif L["kind"] == "mla":
                ctx = self._mla_decode(L, li, normed, pos, slots, bt, seq_lens, n)
                normed, res = self._row_parallel_norm(ctx, L["o"], L["ln2"], res, n)
            else:
                qkv = self._qkv(L, normed, pos, slots, li)
                q3 = qkv.view(n, w.hq + 2 * w.hkv, d)
                ctx = ops.paged_decode_attention(q3[:, : w.hq], self.kv.k[self.kv_of[li]], self.kv.v[self.kv_of[li]], bt, seq_lens, ps,
                                                 self.scale, sinks=L.get("sinks")).reshape(n, -1)  # fmt: skip
                if "gate" in L:
                    ctx = ctx * torch.sigmoid(ops.gemm(normed, L["gate"]).float()).to(ctx.dtype)
                normed, res = self._row_parallel_norm(ctx, L["o"], L["ln2"], res, n, post=L["post_attn_ln"])
            # the norm that follows the MLP is the next layer's input norm (or the final norm)
            next_ln = w.layers[li + 1]["ln1"] if li + 1 < len(w.layers) else w.final_norm
            if "gate_up" in L:
                act = ops.swiglu(_linear(normed, L["gate_up"]))
                normed, res = self._row_parallel_norm(act, L["down"], next_ln, res, n, post=L["post_mlp_ln"])
            else:
                normed, res = ops.rmsnorm(self._post_norm(self._moe(L, normed), L["post_mlp_ln"]), next_ln, cfg.norm_epsilon, res)
        return normed

    def _prepare_reference(self, n):
        st, ds = self._static, self._dev_state
        ps = self.kv.page_size
        init = st["init_mask"][:n].bool()
        for dst, src in (("ids", "init_ids"), ("pos", "init_pos"), ("out_pos", "init_out_pos")):
            ds[dst][:n] = torch.where(init, st[src][:n], ds[dst][:n])
        act = st["active"][:n].bool()
        if "prev" in ds:
            ds["prev"][:n] = torch.where(init, st["init_prev"][:n], ds["prev"][:n])
            ds["prev_eff"][:n] = torch.where(act, ds["prev"][:n], torch.full_like(ds["prev"][:n], -1))
        p = ds["pos"][:n].long()
        slot = st["block_table"][:n].gather(1, (p // ps)[:, None]).squeeze(1).long() * ps + p % ps
        idle = torch.arange(n) % ps
        ds["ids_eff"][:n] = torch.where(act, ds["ids"][:n], torch.zeros_like(ds["ids"][:n]))
        ds["pos_eff"][:n] = torch.where(act, ds["pos"][:n], torch.zeros_like(ds["pos"][:n]))
        ds["seq_lens"][:n] = torch.where(act, ds["pos"][:n] + 1, torch.ones_like(ds["pos"][:n]))
        ds["slots"][:n] = torch.where(act, slot, idle).to(torch.int32)

    @torch.no_grad()
    def decode(self, n: int, filtered: bool, kept_cap: int = 0):
        """One decode step over slots [0, n) (host state must have been uploaded). Under CUDA graphs the
        step is one replay of the bucket that covers ``n``; extra slots are inactive by construction. MoE layers are
        captured too: their expert-sorted layout is built on the device with static shapes. ``last_routed`` holds the
        step's expert choices when ``record_routed`` is set (a buffer of the graph: copy it before the next replay)."""
        if not self.use_cuda_graph:
            *outs, self.last_routed, self.last_logits = self._decode_step(n, filtered, kept_cap)
            return tuple(outs)
        bucket = next(b for b in self.graph_buckets if b >= n)
        key = (bucket, filtered, kept_cap)
        if key not in self.graphs:
            self._capture(bucket, filtered, kept_cap)
        graph, outs, n_kernels = self.graphs[key]
        self.replayed_launches += n_kernels
        graph.replay()
        self.last_routed, self.last_logits = outs[4], outs[5]
        return outs[:4]

    def _capture(self, bucket, filtered, kept_cap):
        """Capture one decode step. Warm-up and capture run with every slot inactive, so they only touch the
        reserved scratch page and leave the device-owned request state unchanged."""
        from slime_b200.ops import _lib

        saved_active = self._static["active"].clone()
        saved_init = self._static["init_mask"].clone()
        self._static["active"].zero_()
        self._static["init_mask"].zero_()
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for _ in range(2):
                self._decode_step(bucket, filtered, kept_cap)
        torch.cuda.current_stream().wait_stream(side)
        g = torch.cuda.CUDAGraph()
        before = _lib.launch_count()
        with torch.cuda.graph(g):
            outs = self._decode_step(bucket, filtered, kept_cap)
        self.graphs[(bucket, filtered, kept_cap)] = (g, outs, _lib.launch_count() - before)
        self._static["active"].copy_(saved_active)
        self._static["init_mask"].copy_(saved_init)

    def drop_graphs(self):
        """Memory tag ``cuda_graph``: captured graphs pin their private pools."""
        self.graphs.clear()


def _extend_attention(q, k_all, v_all, cu_q, cu_k, max_q, max_k, scale, sinks=None):
    """Attention of new tokens over (cached + new) context, causal aligned to the sequence end."""
    if q.is_cuda or sinks is not None:
        from slime_b200.ops import attention

        return attention.segment_attention(q, k_all, v_all, attention.segments_extend(cu_q, cu_k), scale, sinks)
    out = torch.empty_like(q)
    cq, ck = cu_q.tolist(), cu_k.tolist()
    Hq, Hkv = q.shape[1], k_all.shape[1]
    for i in range(len(cq) - 1):
        qs = q[cq[i] : cq[i + 1]].float().transpose(0, 1)
        ks = k_all[ck[i] : ck[i + 1]].float().transpose(0, 1).repeat_interleave(Hq // Hkv, 0)
        vs = v_all[ck[i] : ck[i + 1]].float().transpose(0, 1).repeat_interleave(Hq // Hkv, 0)
        Lq, Lk = qs.shape[1], ks.shape[1]
        att = (qs @ ks.transpose(-1, -2)) * scale
        mask = torch.ones(Lq, Lk, dtype=torch.bool, device=q.device).tril(diagonal=Lk - Lq)
        out[cq[i] : cq[i + 1]] = (att.masked_fill(~mask, float("-inf")).softmax(-1) @ vs).transpose(0, 1).to(q.dtype)
    return out

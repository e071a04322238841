"""Prefill and decode throughput of models with specified layers beside the closest existing model of equal size.

    python bench.py --workload serve [--steps K --warmup W]

Random weights, one GPU, bf16. ``prefill``: one extend pass over packed fresh prompts (logits of the last row of each), tokens
per second. ``decode``: replays of the captured decode step (sampling included) at a fixed batch and context, tokens per
second. Device time by CUDA events around exactly K passes after W warm-up ones; the weights and the cache a pass streams are
several times the L2. The models of a Pefolix pair have the same widths, head counts, layer count and vocabulary; at the context of
``window`` tokens they also read the same keys. A Ledazen pair has the same width, heads, layers and vocabulary; its feed-forward
width is chosen for an equal number of weights in the layers. The Zetizen pairs have the same width, heads, experts and vocabulary, and so
has the mixture pair of Pebodra; its other pair is made like Ledazen's.
Prints one JSON line.
"""

from __future__ import annotations

import dataclasses
import gc
import json

import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.request import Request
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig, get_preset
from slime_b200.models.presets import _ledazen, _pebodra, _pefolix, _zetizen

HYBRID_FF = 14464  # makes the weights of the dense Pebodra layers as many as its partner's
LAYERS = 8  # of the 24 to 36 layers of the models the widths are taken from: per-layer cost is what is compared


def _pairs() -> dict[str, tuple[ModelConfig, ModelConfig]]:
    """name -> (model with specified layers, closest existing model)."""
    dense = get_preset("qwen3-4b")
    dense.num_layers, dense.tie_word_embeddings = LAYERS, False
    small = get_preset("llama-3.2-1b")
    small.num_layers, small.tie_word_embeddings = LAYERS, False
    moe = ModelConfig(num_layers=LAYERS, hidden_size=2048, num_attention_heads=32, num_query_groups=4, kv_channels=128, ffn_hidden_size=6144,
                      vocab_size=151936, rotary_base=1e6, tie_word_embeddings=False, qk_layernorm=True, num_experts=128,
                      moe_ffn_hidden_size=768, moe_router_topk=8, moe_layer_freq=[0, 1] * (LAYERS // 2),
                      moe_shared_expert_intermediate_size=768, moe_shared_expert_gate=True, model_arch="Qwen3MoeForCausalLM")  # fmt: skip
    # delta-net layers with attention in every fourth, against attention beside the delta rule in every fourth
    hybrid = ModelConfig(num_layers=LAYERS, hidden_size=2560, num_attention_heads=32, num_query_groups=8, kv_channels=128, ffn_hidden_size=9216,
                         vocab_size=151936, rotary_base=1e6, tie_word_embeddings=False, qk_layernorm=True, full_attention_interval=4,
                         linear_num_key_heads=16, linear_num_value_heads=32, linear_key_head_dim=128, linear_value_head_dim=128,
                         model_arch="Qwen3_5ForCausalLM")  # fmt: skip
    llama = get_preset("llama-3.2-1b")
    llama.num_layers, llama.tie_word_embeddings = LAYERS, False
    # experts in every layer: grouped attention, and latent attention
    experts = dict(vocab_size=151936, tie_word_embeddings=True, num_experts=128, moe_ffn_hidden_size=768, moe_router_topk=8,
                   moe_shared_expert_intermediate_size=768)  # fmt: skip
    grouped = ModelConfig(num_layers=LAYERS, hidden_size=2048, num_attention_heads=32, num_query_groups=4, kv_channels=128, ffn_hidden_size=6144,
                          rotary_base=1e6, qk_layernorm=True, model_arch="Qwen3MoeForCausalLM", **experts)  # fmt: skip
    latent = ModelConfig(num_layers=LAYERS, hidden_size=2048, num_attention_heads=16, num_query_groups=16, kv_channels=192, ffn_hidden_size=6144,
                         rotary_base=1e6, multi_latent_attention=True, q_lora_rank=768, kv_lora_rank=512, qk_head_dim=128, qk_pos_emb_head_dim=64,
                         v_head_dim=128, model_arch="DeepseekV3ForCausalLM", **experts)  # fmt: skip
    zetizen = lambda kinds: ModelConfig(**_zetizen(kinds, 2048, 151936, 32, 4, 128, 32, 128, 1024, (16, 128, 64, 128, 768, 512), 128, 8, 768, 768))  # noqa: E731,E501
    routed = dataclasses.replace(grouped, tie_word_embeddings=False, moe_shared_expert_intermediate_size=None)
    sizes = ((64, 8, 128, 64), (8, 256, 512), 1024, 4)  # Mamba-2, mLSTM, window, parts of a norm
    return {
        "pebodra-hybrid": (ModelConfig(**_pebodra("MXMA" + "MXMS" * (LAYERS // 4 - 1), 2560, 151936, (32, 8, 64, 128), *sizes, ff=HYBRID_FF)), hybrid),
        "pebodra-moe": (ModelConfig(**_pebodra("maxs" * (LAYERS // 4), 2048, 151936, (32, 4, 64, 128), *sizes, experts=128, top=8, groups=(8, 4),
                                               expert_ff=768)), routed),
        "zetizen-grouped": (zetizen("bc" * (LAYERS // 2)), grouped),
        "zetizen-latent": (zetizen("l" * LAYERS), latent),
        "ledazen-hybrid": (ModelConfig(**_ledazen("dddp" * (LAYERS // 4), 2560, 32, 8, 128, 11776, 151936, 32, 16, 128, 128, 128, 65521)), hybrid),
        "ledazen-d64": (ModelConfig(**_ledazen("p" * LAYERS, 2048, 32, 8, 64, 9984, 128256, 16, 16, 64, 64, 64, 32749)), llama),
        "d128-dense": (ModelConfig(**_pefolix(LAYERS, 2560, 32, 8, 128, 1024, 8, 9728, 151936)), dense),
        "d64-dense": (ModelConfig(**_pefolix(LAYERS, 2048, 32, 8, 64, 1024, 8, 8192, 128256)), small),
        "d128-moe": (ModelConfig(**_pefolix(LAYERS, 2048, 32, 4, 128, 1024, 8, 6144, 151936, every=2, experts=128, top=8, expert_ff=768,
                                            shared_ff=768)), moe),
    }  # fmt: skip


def _timed(fn, steps: int, warmup: int) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for _ in range(steps):
        fn()
    end.record()
    torch.cuda.synchronize()
    return start.elapsed_time(end) / steps


def _place(e: Engine, lengths: list[int]) -> list[Request]:
    out = []
    for i, n in enumerate(lengths):
        r = Request(rid=str(i), input_ids=[(7 * i + j) % 1000 for j in range(n)], sampling=None)
        r.ctx_ids, r.pages = r.input_ids, e.kv.allocator.alloc(-(-n // e.page_size))
        if e.states is not None:
            r.state_slot = e.states.take()
        out.append(r)
    return out


def _give_back(e: Engine, reqs: list[Request]):
    for r in reqs:
        e.kv.allocator.release(r.pages)
        e._give_state(r)


def _prefill_ms(e: Engine, lengths: list[int], steps: int, warmup: int) -> float:
    batch = [(r, len(r.input_ids)) for r in _place(e, lengths)]
    p = e._pack(batch)
    rows = e._to_dev([c - 1 for c in p.cu_q[1:]], torch.long)
    _, dev_in = e._extend_pass(batch, p, rows)
    extend = e._extend_batch(batch) if e.runner.layered or e.runner.recurrent else None
    prev = e._to_dev(p.prev) if e.cfg.bigram else None
    ms = _timed(lambda: e.runner.prefill(*dev_in, p.max_q, p.max_k, rows, True, prev=prev, extend=extend), steps, warmup)
    _give_back(e, [r for r, _ in batch])
    return ms


def _decode_ms(e: Engine, batch: int, context: int, steps: int, warmup: int) -> float:
    """The step is replayed with the slots' positions advancing from ``context``, as generation does."""
    reqs = _place(e, [context + steps + warmup + 2] * batch)
    h = e.runner.host
    for b, r in enumerate(reqs):
        h["active"][b], h["init_mask"][b], h["init_ids"][b], h["init_pos"][b] = 1, 1, 5, context
        h["block_table"][b, : len(r.pages)] = r.pages
        h["state_slot"][b] = r.state_slot or 0
    e.runner.upload_static()
    e.runner.decode(batch, False)
    e.runner.upload_static()  # init records are consumed: from here on the device advances the slots itself
    ms = _timed(lambda: e.runner.decode(batch, False), steps, warmup)
    for b in range(batch):
        e._deactivate(b)
    _give_back(e, reqs)
    return ms


def measure(steps: int = 10, warmup: int = 3, only: str | None = None) -> list[dict]:
    rows = []
    for name, models in _pairs().items():
        if only and only not in name:
            continue
        for cfg in models:
            args = ServerArgs(page_size=64, context_length=8192, max_running_requests=64)
            e = Engine(cfg, args, device="cuda", num_pages=64 * 4200 // 64 + 80)
            e.weights.init_random(0)
            row = dict(pair=name, model=cfg.model_arch, params_b=round(cfg.num_params() / 1e9, 3))
            for label, lengths in (("prefill_8x1024", [1024] * 8), ("prefill_2x4096", [4096] * 2)):
                if cfg.multi_latent_attention and lengths[0] > 1024:
                    continue  # its prompt attention lays every row's context out: more than 100 GB here
                ms = _prefill_ms(e, lengths, steps, warmup)
                row[label] = dict(ms=round(ms, 4), tokens_per_s=round(sum(lengths) / ms * 1e3))
            for label, b, ctx in (("decode_64x1024", 64, 1024), ("decode_64x4096", 64, 4096), ("decode_4x1024", 4, 1024)):
                ms = _decode_ms(e, b, ctx, steps, warmup)
                row[label] = dict(ms=round(ms, 4), tokens_per_s=round(b / ms * 1e3))
            rows.append(row)
            e.shutdown()
            del e
            gc.collect()
            torch.cuda.empty_cache()
    return rows


def main(steps: int, warmup: int, sampler=None, only: str | None = None) -> int:
    from slime_b200.ops import _lib, build

    build.build()
    torch.cuda.set_device(0)
    if sampler is not None:
        sampler.start()
    rows = measure(steps, warmup, only)
    _lib.check_status(torch.device("cuda", 0))
    print(json.dumps({"metric": "serve_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16",
                      "data": "synthetic (random weights and ids)", "config": {"layers": LAYERS, "l2": "inputs larger than L2"}, "rows": rows,
                      "clocks": sampler.stop() if sampler is not None else None}), flush=True)  # fmt: skip
    return 0

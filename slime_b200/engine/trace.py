"""Replay a trace: feed given token ids through a model step by step and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--page-size P] [--max-requests R] < steps.jsonl

A step is one JSON line ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``. The entries of a step run as
one batch (``Engine.feed``): the same extend pass, decode step, CUDA graphs, paged cache and slots that ``Engine.step`` uses
for generation, only the next tokens come from the trace and nothing is sampled from the result. ``want`` lists places
among an entry's tokens; their logits go to ``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``) before ``done <step>``
is printed. ``end`` gives back what the named requests hold. ``--max-tokens`` sizes the page pool.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

KERNEL_GROUP = "serve"  # the part of the kernel library a bf16 / fp32 engine needs


def load_engine(model: str, dtype: str, max_tokens: int, page_size: int, max_requests: int, device=None):
    """An engine for the checkpoint directory ``model`` with a pool of exactly ``max_tokens`` tokens (plus the scratch page)."""
    from slime_b200.checkpoint.hf_loader import SafetensorReader
    from slime_b200.engine.engine import Engine
    from slime_b200.engine.server_args import ServerArgs
    from slime_b200.models.config import ModelConfig

    cfg = ModelConfig.from_hf(model)
    args = ServerArgs(model_path=model, dtype=dtype, page_size=page_size, context_length=max_tokens, max_running_requests=max_requests,
                      disable_radix_cache=True)  # fmt: skip
    engine = Engine(cfg, args, device=device, num_pages=-(-max_tokens // page_size) + 1)
    reader = SafetensorReader(model)
    unknown = engine.update_weights([(n, reader.get(n)) for n in reader.keys() if not n.endswith("_scale_inv")])
    if unknown:
        raise ValueError(f"{model}: tensors this model has no place for: {unknown[:8]}")
    if cfg.layer_specs is not None:
        absent = sorted(set(engine.weights.specified_tensors()) - set(reader.keys()))
        if absent:
            raise ValueError(f"{model}: tensors missing from the checkpoint: {absent[:8]}")
    return engine


class Replay:
    def __init__(self, engine, out: str):
        self.engine, self.out, self.live = engine, out, {}

    def step(self, msg: dict):
        entries = []
        for e in msg["entries"]:
            req = self.live.get(e["id"])
            if req is None:
                req = self.live[e["id"]] = self.engine.open_stream(e["id"])
            entries.append((req, list(e["tokens"]), list(e.get("want") or [])))
        if entries:
            logits = self.engine.feed(entries)
            if logits is not None:
                data = logits.float().contiguous().cpu().numpy().astype("<f4", copy=False)
                path = os.path.join(self.out, f"{msg['step']}.f32")
                with open(path, "wb") as f:
                    f.write(data.tobytes())
            self._check_kernels()
        for rid in msg.get("end") or []:
            req = self.live.pop(rid, None)
            if req is not None:
                self.engine.close_stream(req)

    def _check_kernels(self):
        if self.engine.device.type == "cuda":
            from slime_b200.ops import _lib

            _lib.check_status(self.engine.device)


def main(argv=None) -> int:
    p = argparse.ArgumentParser("trace_run", description=__doc__.split("\n")[0])
    p.add_argument("--model", required=True, help="directory with config.json and *.safetensors")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True, help="directory the logits are written to")
    p.add_argument("--max-tokens", type=int, required=True, help="tokens the live requests hold at most (page pool size)")
    p.add_argument("--page-size", type=int, default=64)
    p.add_argument("--max-requests", type=int, default=4)
    a = p.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    from slime_b200.ops import build

    build.ensure(KERNEL_GROUP)
    import torch

    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a CUDA device")
    replay = Replay(load_engine(a.model, a.dtype, a.max_tokens, a.page_size, a.max_requests, torch.device("cuda", 0)), a.out)
    for line in sys.stdin:
        if line.strip():
            msg = json.loads(line)
            replay.step(msg)
            print(f"done {msg['step']}", flush=True)
    return 0

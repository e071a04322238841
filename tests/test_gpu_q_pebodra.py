"""Pebodra models in the engine on a GPU, bf16 and full precision, against the plain definition (``pebodra_oracle``)."""

import copy
import json
import os
import subprocess
import sys

import pebodra_oracle as O
import pytest
import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig

pytestmark = pytest.mark.gpu
TOL = {"float32": 2e-4, "bfloat16": 0.25}  # of the worst token: rounding the products of the definition to bf16 gives up to half as much
TYPICAL = {"float32": 5e-5, "bfloat16": 0.03}  # of the median token
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CONFIGS = dict(O.CONFIGS, wide=O.model(384, 1000, [  # tensor-core shapes throughout, several key tiles
    (O.ssm(8, 2, 128, 64, 4, 2), O.plain(512)), (O.attn(4, 2, 64, 128, 150, 64, 1e5), O.moe(16, 4, 64, (4, 2))), (O.memory(4, 128, 96), O.moe(8, 2, 128, (2, 1))),
    (O.attn(4, 2, 64, 128, 70, 64, 1e5, diff=0.7, kv_from=1), O.plain(320)), (O.attn(8, 1, 32, 64, 129, 32), None)], norm_groups=4))  # fmt: skip


def make_engine(config, tensors, dtype, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, "dtype": dtype, **kw}
    e = Engine(ModelConfig.from_hf(config), ServerArgs(page_size=page_size, **kw), device="cuda", num_pages=num_pages)
    assert e.dtype == getattr(torch, dtype) and not e.update_weights(tensors.items())
    return e


def weights(config, seed, dtype):
    """bf16 values in either precision; gentler attention where bf16 rounding of q and k would swamp a sharp softmax."""
    t = O.random_tensors(config, seed=seed, sharp=2.5 if dtype == "float32" else 1.0)
    return {k: v.bfloat16() for k, v in t.items()}


def config_of(name, dtype):
    """In bf16 a close call of a router may fall the other way and change a token altogether: use every expert there."""
    config = copy.deepcopy(CONFIGS[name])
    for layer in config["layers"]:
        if dtype == "bfloat16" and layer["mlp"] and layer["mlp"]["kind"] == "moe":
            r = layer["mlp"]["router"]
            r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return config


def agree(got, want, dtype, what=None):
    """Root-mean-square difference of every row, mean taken off, relative to the spread of the logits."""
    d = got.double().cpu() - want
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert float(e.max()) < TOL[dtype] and float(e.median()) < TYPICAL[dtype], (what, float(e.max()), float(e.median()))


@pytest.fixture(params=["bfloat16", "float32"])
def dtype(request):
    return request.param


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding(kernels, name, dtype):
    config = config_of(name, dtype)
    n = 300 if name == "wide" else 120
    tensors, tokens = weights(config, 5, dtype), O.random_tokens(config, n, seed=6)
    want = O.forward(config, tensors, tokens)
    for ps in (16, 64):
        e = make_engine(config, tensors, dtype, page_size=ps)
        for cuts in ([n], [n - 20], [2] * 30, [37, 3, 16, 2, 29]):
            req, at, out = e.open_stream("s"), 0, []
            for c in cuts + [1] * (n - sum(cuts)):
                out.append(e.feed([(req, tokens[at : at + c], list(range(c)))]))
                at += c
            e.close_stream(req)
            agree(torch.cat(out), want, dtype, (ps, cuts))
        assert e.runner.graphs  # single tokens were graph replays


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_mixed_batches_and_reused_slots(kernels, name, dtype):
    config = config_of(name, dtype)
    tensors = weights(config, 7, dtype)
    e = make_engine(config, tensors, dtype, num_pages=1 + 4 * 8, page_size=16)  # four streams of 128 tokens
    lengths = [128, 1, 90, 33, 128, 17, 2, 111, 64]
    want = {i: O.forward(config, tensors, O.random_tokens(config, n, seed=i)) for i, n in enumerate(lengths)}
    g = torch.Generator().manual_seed(1)
    todo, live, got = list(range(len(lengths))), {}, {i: [] for i in want}
    while todo or live:
        while todo and len(live) < 4:
            i = todo.pop(0)
            live[i] = [e.open_stream(str(i)), 0]
        entries, moved = [], []
        for i, (req, at) in live.items():
            c = min([1, 1, 2, 3, 16, 29, 70][int(torch.randint(0, 7, (1,), generator=g))], lengths[i] - at)
            entries.append((req, O.random_tokens(config, lengths[i], seed=i)[at : at + c], list(range(c))))
            moved.append((i, c))
        logits = e.feed(entries).cpu()
        for i, c in moved:
            got[i].append(logits[:c])
            logits = logits[c:]
            live[i][1] += c
            if live[i][1] == lengths[i]:
                e.close_stream(live.pop(i)[0])
    for i in want:
        if len(want[i]) > 30 or dtype == "float32":
            agree(torch.cat(got[i]), want[i], dtype, i)
        assert O.error(torch.cat(got[i]), want[i]) < 2 * TOL[dtype]


@pytest.mark.parametrize("name", ["mixed", "odd", "states"])
def test_greedy_generation(kernels, name, dtype):
    config = config_of(name, dtype)
    tensors = weights(config, 9, dtype)
    e = make_engine(config, tensors, dtype, chunked_prefill_size=13, max_prefill_tokens=21, max_running_requests=3)
    prompts = [O.random_tokens(config, n, seed=20 + n) for n in (37, 1, 18, 50)]
    steps = [12, 30, 9, 25]
    for _ in range(2):  # the second time in used slots, with graphs
        reqs = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
        for p, r in zip(prompts, reqs):
            lp = O.forward(config, tensors, p + r.output_ids).log_softmax(-1)[len(p) - 1 : -1]
            ids = torch.tensor(r.output_ids)[:, None]
            off = (lp.gather(1, ids)[:, 0] - torch.tensor(r.output_logprobs)).abs()
            behind = lp.max(-1).values - lp.gather(1, ids)[:, 0]  # the best token, or a tie with it
            assert float(off.max()) < 4 * TOL[dtype] and float(behind.max()) < 4 * TOL[dtype]
            assert float(off.median()) < 4 * TYPICAL[dtype]
    assert len(e.states.free) == 3


def test_routing_in_bf16(kernels):
    """With a choice of experts: the typical token agrees (a close call may turn a few)."""
    config = CONFIGS["wide"]
    tensors, tokens = weights(config, 7, "bfloat16"), O.random_tokens(config, 200, seed=2)
    want = O.forward(config, tensors, tokens)
    e = make_engine(config, tensors, "bfloat16")
    req = e.open_stream("s")
    got = e.feed([(req, tokens, list(range(200)))]).cpu()
    errors = torch.tensor([O.error(got[t : t + 1], want[t : t + 1]) for t in range(200)])
    assert float(errors.median()) < 0.06


def test_trace_run_program(kernels, tmp_path):
    from safetensors.torch import save_file

    config = CONFIGS["even"]
    tensors = weights(config, 4, "float32")
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_file(tensors, str(tmp_path / "model.safetensors"))
    a = O.random_tokens(config, 70, seed=1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [65, 3]}], "end": []}]
    steps += [{"step": i, "entries": [{"id": "a", "tokens": [a[65 + i]], "want": [0]}], "end": ["a"] if i == 4 else []} for i in range(1, 5)]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=300)  # fmt: skip
    assert r.returncode == 0, r.stderr[-2000:]
    want = O.forward(config, tensors, a)
    rows = [want[[65, 3]]] + [want[65 + i : 66 + i] for i in range(1, 5)]
    for i, w in enumerate(rows):
        got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, config["vocab"])
        assert O.error(got, w) < TOL["float32"]

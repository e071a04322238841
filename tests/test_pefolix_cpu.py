"""Pefolix models in the engine against the plain definition (``pefolix_oracle``), fp32 on the CPU."""

import copy
import json

import pefolix_oracle as O
import pytest
import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig
from slime_b200.ops import grouped, stream
from slime_b200.ops import window_attention as wa

TOL = 6e-5


def make_engine(config, tensors, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, **kw}
    e = Engine(ModelConfig.from_hf(config), ServerArgs(page_size=page_size, **kw), device="cpu", num_pages=num_pages)
    unknown = e.update_weights(tensors.items())
    assert not unknown, unknown
    return e


def feed_all(e, cuts, tokens, req=None):
    """Logits of every token of one stream fed in portions of the sizes ``cuts`` (the rest one by one)."""
    own = req is None
    req = req or e.open_stream("s")
    at, out = 0, []
    cuts = list(cuts) + [1] * (len(tokens) - sum(cuts))
    for n in cuts:
        part = tokens[at : at + n]
        out.append(e.feed([(req, part, list(range(len(part))))]))
        at += n
    if own:
        e.close_stream(req)
    return torch.cat(out)


@pytest.fixture(scope="module", params=sorted(O.CONFIGS))
def case(request):
    config = O.CONFIGS[request.param]
    tensors = O.random_tensors(config, seed=5)
    tokens = O.random_tokens(config, 75, seed=6)
    return config, tensors, tokens, O.forward(config, tensors, tokens)


# ------------------------------------------------------------------------------------ mechanisms alone
def test_layer_norm_and_residual():
    g = torch.Generator().manual_seed(0)
    y, res, w1, w2 = (torch.randn(*s, generator=g) for s in ((6, 50), (6, 50), (50,), (50,)))
    y = y * 4 + 3  # a mean that a norm without centring would keep
    want = res + O.layer_norm(y, w1, 0.05)
    h, out = stream.stream_norm(y, res.clone(), w2, 0.05, kind="layer", post_w=w1)
    torch.testing.assert_close(out, want)
    torch.testing.assert_close(h, O.layer_norm(want, w2, 0.05))
    assert float((stream.stream_norm(y, None, w2, 0.05, kind="rms")[0] - O.layer_norm(y, w2, 0.05)).abs().max()) > 0.1


def test_activations():
    x = torch.randn(9, 24, generator=torch.Generator().manual_seed(1)) * 3
    torch.testing.assert_close(stream.feed_forward_act(x, "gelu_tanh", True), O.gelu_tanh(x[:, :12]) * x[:, 12:])
    torch.testing.assert_close(stream.feed_forward_act(x, "relu2", False), O.relu_squared(x))


@pytest.mark.parametrize("experts,top,shared", [(7, 2, True), (5, 1, False), (4, 4, True)])
def test_mixture(experts, top, shared):
    g = torch.Generator().manual_seed(experts)
    h, router, sg = torch.randn(11, 20, generator=g), torch.randn(experts, 20, generator=g), torch.randn(1, 20, generator=g)
    ups, downs = torch.randn(experts, 12, 20, generator=g), torch.randn(experts, 20, 12, generator=g)
    sh = (torch.randn(9, 20, generator=g), torch.randn(20, 9, generator=g)) if shared else None
    want = O.mixture(h, router, list(zip(ups, downs)), top, sh, sg if shared else None)
    logits = h @ torch.cat([router, sg]).t()
    probs, idx = grouped.route_topk(logits[:, :experts], top, renorm=False)
    lay = grouped.DeviceLayout(idx, experts)
    rows = grouped.grouped_gemm(stream.feed_forward_act(grouped.grouped_gemm(lay.pad(h), ups, lay), "relu2", False), downs, lay)
    e = stream.ExpertSum(rows, lay.slot_dest, probs)
    if shared:
        e.shared, e.gate = stream.feed_forward_act(h @ sh[0].t(), "relu2", False) @ sh[1].t(), logits[:, experts]
    torch.testing.assert_close(stream.combine(e), want, atol=1e-4, rtol=1e-4)
    weight, index = O.route(h, router, top)
    assert torch.equal(index.sort(-1).values, idx.sort(-1).values) and (top == experts or float(weight.sum(-1).max()) < 1)


@pytest.mark.parametrize("size,keep", [(1, 0), (7, 0), (7, 3), (16, 16), (5, 40), (100, 2)])
def test_attention(size, keep):
    spec = O.attn(6, 2, 16, 24, size, keep, scale=0.4)
    g = torch.Generator().manual_seed(size)
    T, ps, D = 53, 16, 30
    h = torch.randn(T, D, generator=g)
    wq, wk, wv, wo = (torch.randn(*s, generator=g) * 0.5 for s in ((96, D), (32, D), (48, D), (D, 144)))
    want = O.attention(h, wq, wk, wv, wo, spec)
    kc, vc, pages = torch.zeros(6 * ps, 2, 16), torch.zeros(6 * ps, 2, 24), [4, 1, 5, 2]
    slots = torch.tensor([pages[p // ps] * ps + p % ps for p in range(T)], dtype=torch.int32)
    stream.kv_scatter(h @ wk.t(), h @ wv.t(), slots, kc, vc)
    q = (h @ wq.t()).view(T, 6, 16)
    slopes = torch.tensor(ModelConfig.from_hf(O.model(D, 9, [(spec, None)])).layer_specs[0].mixer.slopes())
    torch.testing.assert_close(slopes, torch.tensor(O.distance_slopes(6)))
    batch = wa.ExtendBatch.build([pages], [0], [T], ps, "cpu")
    got = wa.window_extend(q, kc, vc, batch, 0.4, size, keep, slopes).flatten(1) @ wo.t()
    torch.testing.assert_close(got, want, atol=2e-4, rtol=2e-4)
    for t in (0, 1, size - 1, size, 17, T - 1):
        if 0 <= t < T:
            one = torch.tensor([t], dtype=torch.int32)
            got = wa.window_decode(q[t : t + 1], kc, vc, batch.block_table, one + 1, one, ps, 0.4, size, keep, slopes)
            torch.testing.assert_close((got.flatten(1) @ wo.t())[0], want[t], atol=2e-4, rtol=2e-4)


def test_tile_table_covers_every_row_once():
    batch = wa.ExtendBatch.build([[1, 2], [3], [4, 5, 6]], [3, 0, 40], [20, 1, 7], 16, "cpu")
    for tokens in (1, 6, 128):
        rows = []
        for row0, n, pos, r in batch.tiles(tokens).tolist():
            assert 1 <= n <= tokens
            for k in range(n):
                assert int(batch.row_req[row0 + k]) == r and int(batch.positions[row0 + k]) == pos + k
                rows.append(row0 + k)
        assert rows == list(range(28))
    assert wa.tile_tokens(6, 2) == 42 and wa.tile_tokens(128, 1) == 1 and wa.tile_tokens(129, 1) == 0


# ------------------------------------------------------------------------------------ whole models
def test_prompt_portions_and_decoding_agree_with_the_definition(case):
    config, tensors, tokens, want = case
    layers = []
    O.forward(config, tensors, tokens[:20], torch.float64, layers)
    for ps in (4, 16):
        e = make_engine(config, tensors, page_size=ps)
        seen = {}
        e.runner.stream_hook = lambda li, res: seen.setdefault(li, res.clone())
        req = e.open_stream("a")
        e.feed([(req, tokens[:20], [])])
        e.close_stream(req)
        for li, x in enumerate(layers):
            assert float((seen[li].double() - x).abs().max()) < 1e-4 * float(x.abs().max()), li
        e.runner.stream_hook = None
        free = len(e.kv.allocator.free)
        for cuts in ([75], [], [2] * 37, [3, 16, 5, 2, 30], [64, 11], [7, 1, 1, 13, 2, 2, 41]):
            assert O.error(feed_all(e, cuts, tokens), want) < TOL, cuts
            assert len(e.kv.allocator.free) == free and len(e.free_slots) == 4
        assert e.stats["decode_steps"] > 70  # single tokens take the decode step


def test_unequal_batches_equal_each_request_alone(case):
    """Portions beside single tokens, streams that pause, streams that end and whose pages and slots the next ones take."""
    config, tensors, _, _ = case
    e = make_engine(config, tensors, num_pages=1 + 4 * 4, page_size=16)  # room for four streams of 64 tokens, no more
    g = torch.Generator().manual_seed(9)
    lengths = [64, 1, 33, 50, 17, 64, 40, 2, 61, 48]
    want = {i: O.forward(config, tensors, O.random_tokens(config, n, seed=i)) for i, n in enumerate(lengths)}
    todo, live, got = list(range(len(lengths))), {}, {i: [] for i in want}
    while todo or live:
        while todo and len(live) < 4:
            i = todo.pop(0)
            live[i] = [e.open_stream(str(i)), 0]
        entries, moved = [], []
        for i, (req, at) in live.items():
            if len(live) > 1 and int(torch.randint(0, 4, (1,), generator=g)) == 0:
                continue  # left out of this step
            n = min([1, 1, 2, 3, 16, 29][int(torch.randint(0, 6, (1,), generator=g))], lengths[i] - at)
            part = O.random_tokens(config, lengths[i], seed=i)[at : at + n]
            entries.append((req, part, list(range(n))))
            moved.append((i, n))
        if not entries:
            continue
        logits = e.feed(entries)
        for i, n in moved:
            got[i].append(logits[:n])
            logits = logits[n:]
            live[i][1] += n
            if live[i][1] == lengths[i]:
                e.close_stream(live.pop(i)[0])
    for i in want:
        assert O.error(torch.cat(got[i]), want[i]) < TOL, i
    assert len(e.kv.allocator.free) == 16


def test_greedy_generation_through_the_scheduler(case):
    config, tensors, _, _ = case
    prompts = [O.random_tokens(config, n, seed=20 + n) for n in (37, 1, 18, 50, 5)]
    steps = [12, 30, 9, 4, 40]
    e = make_engine(config, tensors, chunked_prefill_size=13, max_prefill_tokens=21, max_running_requests=3)
    reqs = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
    for p, n, r in zip(prompts, steps, reqs):
        assert len(r.output_ids) == n
        lp = O.forward(config, tensors, p + r.output_ids).log_softmax(-1)
        picks = lp[len(p) - 1 : -1]
        assert torch.equal(picks.argmax(-1), torch.tensor(r.output_ids))
        want = picks.gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
        assert float((want - torch.tensor(r.output_logprobs)).abs().max()) < 1e-3
    # the same prompts again: whole pages come from the prefix cache, the answers are the same
    again = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
    assert [r.output_ids for r in again] == [r.output_ids for r in reqs] and again[0].num_cached_tokens == 32
    # prompt log-probs (one pass over every position)
    r = e.generate([prompts[0]], [dict(max_new_tokens=0)], logprob_start_len=0)[0]
    lp = O.forward(config, tensors, prompts[0]).log_softmax(-1)[:-1].gather(1, torch.tensor(prompts[0][1:])[:, None])[:, 0]
    assert float((lp - torch.tensor(r.input_logprobs[1:])).abs().max()) < 1e-3


def test_generation_under_page_pressure(case):
    config, tensors, _, _ = case
    prompts = [O.random_tokens(config, 30, seed=40 + i) for i in range(3)]
    sp = [dict(max_new_tokens=40, temperature=0, ignore_eos=True)] * 3
    roomy = make_engine(config, tensors, num_pages=64, page_size=8).generate(prompts, sp)
    tight = make_engine(config, tensors, num_pages=1 + 16, page_size=8, disable_radix_cache=True)  # 128 tokens for 3 x 70
    assert [r.output_ids for r in tight.generate(prompts, sp)] == [r.output_ids for r in roomy]


@pytest.mark.parametrize("name", ["mixed", "equal"])
def test_long_decoding_slides_the_window(name):
    config = O.CONFIGS[name]
    tensors, tokens = O.random_tensors(config, seed=2), O.random_tokens(config, 230, seed=3)
    want = O.forward(config, tensors, tokens)
    assert O.error(feed_all(make_engine(config, tensors), [9], tokens), want) < TOL


MISTAKES = {
    "window one longer": lambda c: [x["mixer"]["mask"].update(size=x["mixer"]["mask"]["size"] + 1) for x in c["layers"]],
    "window one shorter": lambda c: [x["mixer"]["mask"].update(size=x["mixer"]["mask"]["size"] - 1) for x in c["layers"]],
    "one token more kept": lambda c: [x["mixer"]["mask"].update(keep_first=x["mixer"]["mask"]["keep_first"] + 1) for x in c["layers"]],
    "nothing kept": lambda c: [x["mixer"]["mask"].update(keep_first=0) for x in c["layers"]],
    "scale": lambda c: [x["mixer"].update(scale=x["mixer"]["scale"] * 1.02) for x in c["layers"]],
    "eps": lambda c: c["norm"].update(eps=c["norm"]["eps"] * 10),
    "an expert less": lambda c: [x["mlp"]["router"].update(top=x["mlp"]["router"]["top"] - 1) for x in c["layers"] if x["mlp"]["kind"] == "moe"],
    "no shared expert": lambda c: [x["mlp"].pop("shared", None) for x in c["layers"] if x["mlp"]["kind"] == "moe"],
}  # fmt: skip


@pytest.mark.parametrize("mistake", sorted(MISTAKES) + ["slopes", "value heads"])
def test_a_mistake_in_the_definition_shows(mistake, monkeypatch):
    """The comparison is sharp: with one thing wrong in the definition the engine no longer agrees with it."""
    config = copy.deepcopy(O.CONFIGS["odd"])
    config["layers"][1]["mlp"]["router"]["top"] = 2
    tensors, tokens = O.random_tensors(config, seed=1), O.random_tokens(config, 60, seed=1)
    got = feed_all(make_engine(config, tensors), [31, 2], tokens)
    assert O.error(got, O.forward(config, tensors, tokens)) < TOL
    wrong = copy.deepcopy(config)
    if mistake == "slopes":
        monkeypatch.setattr(O, "distance_slopes", lambda heads: [2.0 ** (-8.0 * h / heads) for h in range(heads)])
    elif mistake == "value heads":
        tensors = dict(tensors, **{"l1.mix.v": tensors["l1.mix.v"].roll(22, 0)})
    else:
        MISTAKES[mistake](wrong)
    assert O.error(got, O.forward(wrong, tensors, tokens)) > 5 * TOL


# ------------------------------------------------------------------------------------ configuration, loading, cache
def test_configuration_round_trip():
    for config in O.CONFIGS.values():
        cfg = ModelConfig.from_hf(config)
        assert cfg.to_hf_dict() == config
        assert cfg.num_params() == sum(v.numel() for v in O.random_tensors(config).values())
        assert ModelConfig.from_hf(json.loads(json.dumps(cfg.to_hf_dict()))) == cfg
    bad = copy.deepcopy(O.CONFIGS["single"])
    bad["layers"][0]["type"] = "recurrent"
    with pytest.raises(ValueError, match="mixer"):
        ModelConfig.from_hf(bad)


def test_loader_refuses_what_the_model_does_not_have():
    config = O.CONFIGS["mixed"]
    e = make_engine(config, O.random_tensors(config))
    z = torch.zeros(96, 96)
    for name in ("l1.norm2", "l1.mlp.up", "l0.mlp.router", "l2.mlp.gate", "l2.mlp.e7.up", "l3.mlp.shared.up", "l2.mlp.e0.gate", "l5.norm1", "x"):
        assert e.update_weights([(name, z)]) == [name]
    with pytest.raises(ValueError, match="shape"):
        e.update_weights([("l0.mix.o", z)])
    assert set(e.weights.specified_tensors()) == set(O.random_tensors(config))


def test_trainer_says_that_it_cannot_train_this():
    from slime_b200.models.gpt import GPTModel

    with pytest.raises(NotImplementedError, match="rollout engine only"):
        GPTModel(ModelConfig.from_hf(O.CONFIGS["single"]), dtype=torch.float32, device="cpu")


@pytest.mark.parametrize("name", ["mixed", "equal"])
def test_hand_over_and_host_tier(name):
    """Keys and values travel between engines, and evicted pages come back from host memory, for layers of equal and of
    different geometry."""
    config = O.CONFIGS[name]
    tensors, prompt = O.random_tensors(config, seed=8), O.random_tokens(config, 45, seed=8)
    sp = dict(max_new_tokens=10, temperature=0, ignore_eos=True)
    a, b = make_engine(config, tensors), make_engine(config, tensors)
    assert a.kv.uniform == (name == "equal")
    want = a.generate([prompt], [sp])[0]
    pre = a.generate([prompt], [sp], prefill_only=True)[0]
    with pytest.raises(ValueError, match="does not fit"):
        b.import_request(prompt[:-1], pre.output_ids[0], 0.0, pre.kv_export, sp)
    r = b.import_request(prompt, pre.output_ids[0], pre.output_logprobs[0], pre.kv_export, sp)
    while not r.finished():
        b.step()
    assert r.output_ids == want.output_ids
    small = make_engine(config, tensors, num_pages=9, enable_hierarchical_cache=True, hicache_ratio=4.0)
    small.generate([prompt], [sp])
    for i in range(3):
        small.generate([O.random_tokens(config, 60, seed=60 + i)], [sp])
    again = small.generate([prompt], [sp])[0]
    assert again.output_ids == want.output_ids and small.kv.allocator.host_tier.hits > 0


def test_replay_writes_the_wanted_logits(tmp_path):
    from safetensors.torch import save_file

    from slime_b200.engine import trace

    config = O.CONFIGS["mixed"]
    tensors = O.random_tensors(config, seed=4)
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_file(tensors, str(tmp_path / "model.safetensors"))
    r = trace.Replay(trace.load_engine(str(tmp_path), "float32", 128, 64, 4, torch.device("cpu")), str(tmp_path))
    assert len(r.engine.kv.allocator.free) == 2  # 128 tokens in pages of 64; the scratch page is extra
    a, b = O.random_tokens(config, 40, seed=1), O.random_tokens(config, 9, seed=2)
    r.step({"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [32, 0]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []})
    r.step({"step": 1, "entries": [{"id": "a", "tokens": a[33:34], "want": []}], "end": []})
    r.step({"step": 2, "entries": [{"id": "b", "tokens": b[1:], "want": [7]}, {"id": "a", "tokens": a[34:35], "want": [0]}], "end": ["a", "b"]})
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 203)  # noqa: E731
    la, lb = O.forward(config, tensors, a), O.forward(config, tensors, b)
    assert O.error(read(0), la[[32, 0]]) < TOL and O.error(read(2), torch.stack([lb[8], la[34]])) < TOL
    assert not (tmp_path / "1.f32").exists() and not r.live and len(r.engine.free_slots) == 4
    with pytest.raises(ValueError, match="context length"):
        r.step({"step": 3, "entries": [{"id": "c", "tokens": a * 4, "want": []}], "end": []})


def _rank_main(rank, port, config, tensors, tokens, want, ep):
    import torch.distributed as dist

    torch.set_num_threads(1)
    dist.init_process_group("gloo", init_method=f"tcp://127.0.0.1:{port}", rank=rank, world_size=2)
    args = ServerArgs(page_size=16, max_running_requests=4, context_length=128, ep_size=ep)
    e = Engine(ModelConfig.from_hf(config), args, device="cpu", num_pages=16, tp_group=dist.group.WORLD, tp_size=2, tp_rank=rank)
    assert not e.update_weights(tensors.items())
    assert O.error(feed_all(e, [17, 2, 20], tokens), want) < TOL
    dist.destroy_process_group()


@pytest.mark.parametrize("ep", [1, 2])
def test_two_tensor_parallel_ranks(ep):
    import socket

    config = O.model(48, 70, [(O.attn(4, 2, 16, 24, 14, 3), O.dense(40)), (O.attn(6, 2, 8, 16, 30, 0), O.moe(24, 6, 3, shared=20)),
                              (O.attn(2, 2, 16, 16, 9, 9), O.moe(16, 4, 1))])  # fmt: skip
    tensors, tokens = O.random_tensors(config, seed=3), O.random_tokens(config, 44, seed=3)
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    want = O.forward(config, tensors, tokens)
    torch.multiprocessing.spawn(_rank_main, args=(port, config, tensors, tokens, want, ep), nprocs=2)
    with pytest.raises(ValueError, match="divide"):
        cfg = ModelConfig.from_hf(O.CONFIGS["odd"])
        Engine(cfg, ServerArgs(), device="cpu", num_pages=4, tp_size=2)

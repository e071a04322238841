"""Ledazen models in the engine against the plain definition (``ledazen_oracle``), fp32 on the CPU."""

import copy
import json

import ledazen_oracle as O
import pytest
import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.projections import LayerProjections
from slime_b200.engine.server_args import ServerArgs
from slime_b200.engine.state_cache import OutOfStateSlots, RecurrentStates
from slime_b200.models.config import ModelConfig
from slime_b200.models.layer_spec import DeltaSpec, LayerSpec
from slime_b200.ops import delta, stream
from slime_b200.ops import window_attention as wa

TOL = 1e-4


def make_engine(config, tensors, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, **kw}
    e = Engine(ModelConfig.from_hf(config, O.shapes(tensors)), ServerArgs(page_size=page_size, **kw), device="cpu", num_pages=num_pages)
    unknown = e.update_weights(tensors.items())
    assert not unknown, unknown
    return e


def feed_all(e, cuts, tokens):
    """Logits of every token of one stream fed in portions of the sizes ``cuts`` (the rest one by one)."""
    req, at, out = e.open_stream("s"), 0, []
    for n in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        part = tokens[at : at + n]
        out.append(e.feed([(req, part, list(range(len(part))))]))
        at += n
    e.close_stream(req)
    return torch.cat(out)


@pytest.fixture(scope="module", params=sorted(O.CONFIGS))
def case(request):
    config = O.CONFIGS[request.param]
    tensors = O.random_tensors(config, seed=5)
    tokens = O.random_tokens(config, 75, seed=6)
    return config, tensors, tokens, O.forward(config, tensors, tokens)


# ------------------------------------------------------------------------------------ mechanisms alone
def test_bigram_rows_and_the_norm_around_one():
    g = torch.Generator().manual_seed(0)
    embed, table, w = (torch.randn(*s, generator=g) for s in ((50, 24), (18, 24), (24,)))
    tokens = [3, 49, 3, 3, 0, 17]
    rows = O.bigram_rows(tokens, 17, 1000003, 77)  # products beyond 32 bits
    assert rows[0] == 17 and len(set(rows)) > 3
    ids = torch.tensor(tokens, dtype=torch.int32)
    pair = stream.PairTable(table, ids, torch.tensor([-1] + tokens[:-1], dtype=torch.int32), 1000003, 77)
    assert pair.rows().tolist() == rows
    h, res = stream.stream_norm(embed, None, w, 0.05, ids=ids, offset=1.0, pair=pair)
    torch.testing.assert_close(res, embed[tokens] + table[rows])
    torch.testing.assert_close(h, O.rms_around_one(res, w, 0.05))


@pytest.mark.parametrize("dims", [0, 2, 10, 16])
def test_query_and_key_norm_rotation_and_sink(dims):
    spec, D, T, ps = O.attn(6, 2, 16, 24, dims, base=50.0, scale=0.7), 30, 53, 16
    g = torch.Generator().manual_seed(dims)
    W = {n: torch.randn(*s, generator=g) * 0.4 for n, s in (("q", (96, D)), ("k", (32, D)), ("v", (48, D)), ("o", (D, 144)),
                                                            ("q.norm", (16,)), ("k.norm", (16,)))}  # fmt: skip
    h = torch.randn(T, D, generator=g)
    want = O.attention(h, lambda n: W[n], spec, 1e-3)
    kc, vc, pages = torch.zeros(6 * ps, 2, 16), torch.zeros(6 * ps, 2, 24), [4, 1, 5, 2]
    slots = torch.tensor([pages[p // ps] * ps + p % ps for p in range(T)], dtype=torch.int32)
    batch = wa.ExtendBatch.build([pages], [0], [T], ps, "cpu")
    q = stream.place_heads(*(h @ W[n].t() for n in "qkv"), slots, kc, vc, q_norm=W["q.norm"], k_norm=W["k.norm"], eps=1e-3,
                           table=stream.rotary_table(64, dims, 50.0) if dims else None, positions=batch.positions)
    sinks = torch.zeros(6)
    got = wa.window_extend(q, kc, vc, batch, 0.7, sinks=sinks, out_scale=0.25).flatten(1) @ W["o"].t()
    torch.testing.assert_close(got, 0.25 * want, atol=2e-4, rtol=2e-4)
    out = torch.zeros(1, 150)
    for t in (0, 1, 15, 16, T - 1):
        one = torch.tensor([t], dtype=torch.int32)
        wa.window_decode(q[t : t + 1], kc, vc, batch.block_table, one + 1, one, ps, 0.7, sinks=sinks, out=out[:, 3:147])
        torch.testing.assert_close((out[:, 3:147] @ W["o"].t())[0], want[t], atol=2e-4, rtol=2e-4)
    assert float((wa.window_extend(q, kc, vc, batch, 0.7).flatten(1) @ W["o"].t() - want).abs().max()) > 1e-2  # the sink counts


def test_rotation_of_halves_is_the_other_layout():
    x, table = torch.randn(5, 2, 12), stream.rotary_table(9, 8, 30.0)
    pos = torch.tensor([0, 3, 1, 8, 5])
    perm = [0, 2, 4, 6, 1, 3, 5, 7, 8, 9, 10, 11]  # pairs next to each other -> half apart
    torch.testing.assert_close(stream._turn(x, table, pos, True)[..., perm], stream._turn(x[..., perm], table, pos, False))


def _rule_case(H, G, D, DV, taps, per_channel, T, seed=0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x = delta.DeltaInputs(r(T, G * D), r(T, G * D), r(T, H * DV), r(T, H * D if per_channel else H) - 2, r(T, H), r(2 * G * D + H * DV, taps) * 0.6,
                          r(H) * 0.5, r(H * D if per_channel else H))  # fmt: skip
    y = O.short_conv(torch.cat([x.q, x.k, x.v], 1), x.conv)
    q, k, v = y[:, : G * D].view(T, G, D), y[:, G * D : 2 * G * D].view(T, G, D), y[:, 2 * G * D :].view(T, H, DV)
    q, k = O.unit(q) * D**-0.5, O.unit(k)
    z = O.softplus(x.a + x.dt_bias)
    z = z.view(T, H, D) if per_channel else z[:, :, None].expand(T, H, D)
    decay = torch.exp(-torch.exp(x.A_log)[None, :, None] * z)
    want = torch.stack([O.delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], decay[:, h], torch.sigmoid(x.b[:, h])) for h in range(H)], 1)
    return x, want


def _rows(x, lo, hi):
    return delta.DeltaInputs(*(t[lo:hi] for t in (x.q, x.k, x.v, x.a, x.b)), x.conv, x.A_log, x.dt_bias)


@pytest.mark.parametrize("per_channel", [False, True])
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_delta_rule_in_portions_and_steps(per_channel, taps):
    H, G, D, DV, T = 4, 2, 6, 5, 40
    x, want = _rule_case(H, G, D, DV, taps, per_channel, T, seed=taps)
    z, w = torch.randn(T, H * DV), torch.randn(DV)
    state, ring = torch.full((3, H, D, DV), 9.0), torch.full((3, taps, 2 * G * D + H * DV), 9.0)  # what an earlier request left
    for cuts in ([40], [2] * 20, [3, 1, 2, 17, 9, 8], [1] * 40):
        at, got = 0, []
        for n in cuts:
            if n == 1 and at > 0:
                one = lambda v: torch.tensor([0, v, 0], dtype=torch.int32)  # noqa: E731
                part = _rows(x, at, at + 1)
                pad = delta.DeltaInputs(*(t.expand(3, -1) for t in (part.q, part.k, part.v, part.a, part.b)), x.conv, x.A_log, x.dt_bias)
                before = state[[0, 2]].clone()
                y = delta.delta_step(pad, state, ring, one(1), one(1), one(at), z[at : at + 1].expand(3, -1), w, "silu", 0.01, 0.5)
                assert torch.equal(state[[0, 2]], before) and float(y[[0, 2]].abs().max()) == 0
                gate = O.silu(z[at]).view(H, DV)
                torch.testing.assert_close(y[1].view(H, DV), 0.5 * O.rms(want[at], 0.01) * w * gate, atol=2e-4, rtol=2e-4)
                got.append(want[at : at + 1])
            else:
                batch = wa.ExtendBatch.build([[0]], [at], [n], 64, "cpu", state_slots=[1])
                got.append(delta.delta_extend(_rows(x, at, at + n), state, ring, batch))
            at += n
        torch.testing.assert_close(torch.cat(got), want, atol=2e-4, rtol=2e-4)
    torch.testing.assert_close(delta.head_gate(want, z, w, "sigmoid", 0.01), (O.rms(want, 0.01) * w * torch.sigmoid(z).view(T, H, DV)).flatten(1))


def test_two_portions_of_different_requests_in_one_pass():
    H, G, D, DV, taps = 3, 3, 5, 4, 4
    (xa, wa_), (xb, wb) = (_rule_case(H, G, D, DV, taps, True, 20, seed=s) for s in (1, 1))
    xb = delta.DeltaInputs(*(t.flip(0) for t in (xb.q, xb.k, xb.v, xb.a, xb.b)), xb.conv, xb.A_log, xb.dt_bias)
    state, ring = torch.zeros(2, H, D, DV), torch.zeros(2, taps, 2 * G * D + H * DV)
    both = lambda a, b: delta.DeltaInputs(*(torch.cat([s, t]) for s, t in zip((a.q, a.k, a.v, a.a, a.b), (b.q, b.k, b.v, b.a, b.b))), xa.conv, xa.A_log, xa.dt_bias)  # noqa: E731,E501
    first = delta.delta_extend(both(_rows(xa, 0, 7), _rows(xb, 0, 12)), state, ring, wa.ExtendBatch.build([[0], [1]], [0, 0], [7, 12], 16, "cpu", state_slots=[1, 0]))
    second = delta.delta_extend(both(_rows(xb, 12, 20), _rows(xa, 7, 20)), state, ring, wa.ExtendBatch.build([[1], [0]], [12, 7], [8, 13], 16, "cpu", state_slots=[0, 1]))
    torch.testing.assert_close(torch.cat([first[:7], second[8:]]), wa_, atol=1e-4, rtol=1e-4)
    alone, _ = torch.zeros(1, H, D, DV), None
    want = delta.delta_extend(xb, alone, torch.zeros(1, taps, 2 * G * D + H * DV), wa.ExtendBatch.build([[0]], [0], [20], 32, "cpu", state_slots=[0]))
    torch.testing.assert_close(torch.cat([first[7:], second[:8]]), want, atol=1e-4, rtol=1e-4)


def test_state_slots():
    s = RecurrentStates([(2, 3, 4, 20, 4), (1, 8, 8, 24, 2)], 2, torch.float32, torch.device("cpu"))
    assert [tuple(x.shape) for x in s.state + s.ring] == [(2, 2, 3, 4), (2, 1, 8, 8), (2, 4, 20), (2, 2, 24)]
    a, b = s.take(), s.take()
    with pytest.raises(OutOfStateSlots):
        s.take()
    s.give(b)
    assert s.take() == b and a != b
    s.give(a)
    with pytest.raises(AssertionError):
        s.give(a)


def test_fused_matrices_hold_every_tensor_once():
    for config in O.CONFIGS.values():
        tensors = O.random_tensors(config)
        for i, spec in enumerate(ModelConfig.from_hf(config, O.shapes(tensors)).layer_specs):
            lay = LayerProjections(spec)
            want = {k[len(f"l{i}.") :]: v for k, v in O.shapes(tensors).items() if k.startswith(f"l{i}.") and not k.endswith("norm1")}
            assert lay.tensors(config["width"]) == want
            for ranges, total in ((lay.ins, lay.in_rows), (lay.outs, lay.out_cols)):
                used = sorted(ranges.values())
                assert all(a % 8 == 0 for a, _ in used) and all(a + n <= b for (a, n), (b, _) in zip(used, used[1:] + [(total, 0)]))


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
        for cuts in ([75], [], [2] * 37, [3, 16, 5, 2, 30], [7, 1, 1, 13, 2, 2, 41]):
            assert O.error(feed_all(e, cuts, tokens), want) < TOL, cuts
            assert len(e.kv.allocator.free) == free and len(e.free_slots) == len(e.states.free) == 4
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
    assert len(e.kv.allocator.free) == 16 and len(e.states.free) == 4


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
    # the same prompts again, in used slots; a state at a page's end is not kept, so nothing comes from the prefix cache
    again = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
    assert [r.output_ids for r in again] == [r.output_ids for r in reqs] and again[0].num_cached_tokens == 0
    assert len(e.states.free) == 3
    r = e.generate([prompts[0]], [dict(max_new_tokens=0)], logprob_start_len=0)[0]  # prompt log-probs
    lp = O.forward(config, tensors, prompts[0]).log_softmax(-1)[:-1].gather(1, torch.tensor(prompts[0][1:])[:, None])[:, 0]
    assert float((lp - torch.tensor(r.input_logprobs[1:])).abs().max()) < 1e-3


def test_generation_under_page_pressure_and_after_an_abort(case):
    config, tensors, _, _ = case
    prompts = [O.random_tokens(config, 30, seed=40 + i) for i in range(3)]
    sp = [dict(max_new_tokens=40, temperature=0, ignore_eos=True)] * 3
    roomy = make_engine(config, tensors, num_pages=64, page_size=8).generate(prompts, sp)
    tight = make_engine(config, tensors, num_pages=1 + 16, page_size=8)  # 128 tokens for 3 x 70: requests are retracted
    waiting = [tight.add_request(p, s) for p, s in zip(prompts, sp)]
    for _ in range(7):
        tight.step()
    tight.abort(abort_all=True)
    assert len(tight.states.free) == 4 and all(r.finished() for r in waiting)
    assert [r.output_ids for r in tight.generate(prompts, sp)] == [r.output_ids for r in roomy]
    tight.release_memory_occupation(["kv_cache"])
    assert not tight.states.state
    tight.resume_memory_occupation(["kv_cache"])
    assert tight.generate(prompts[:1], sp[:1])[0].output_ids == roomy[0].output_ids


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding(name):
    config = O.CONFIGS[name]
    tensors, tokens = O.random_tensors(config, seed=2), O.random_tokens(config, 220, seed=3)
    want = O.forward(config, tensors, tokens)
    assert O.error(feed_all(make_engine(config, tensors), [9], tokens), want) < TOL


@pytest.mark.parametrize("cut", [0, 60])
def test_a_key_far_back_is_found(cut):
    """One token's query matches one far token's key in every head and nothing else does: the answer must move with the value
    stored there, whether the prompt is one portion or the query is a decoded token."""
    config = O.model(48, 40, (19, 3, 5), [(O.both(O.attn(4, 2, 16, 16, 4, scale=4.0), O.rule(2, 1, 8, 8, 3)), 32)])
    tensors = O.random_tensors(config, seed=3, sharp=1.0)
    n, far = 150, 17
    # coordinate 0 of the stream marks token 38, coordinate 1 token 39; unturned coordinates of k and q read them
    for name in ("embed", "bigram"):
        tensors[name][:, :2] = 0.0
    tensors["embed"][38, 0] = tensors["embed"][39, 1] = 30.0
    for mark, x in enumerate("kq"):
        w = tensors[f"l0.mix.left.{x}"].view(-1, 16, 48)
        w[:, :, :2] = 0.0
        w[:, 12, mark] = 20.0
        tensors[f"l0.mix.left.{x}.norm"] = torch.ones(16)
    tokens = [t % 38 for t in O.random_tokens(config, n, seed=1)]
    tokens[far], tokens[-1] = 38, 39
    want = O.forward(config, tensors, tokens)
    other = list(tokens)
    other[far] = 5
    assert O.error(O.forward(config, tensors, other)[-1:], want[-1:]) > 0.2  # the far key decides
    for ps in (4, 64):
        e = make_engine(config, tensors, page_size=ps, num_pages=256 // ps + 1)
        assert O.error(feed_all(e, [n - cut], tokens), want) < TOL


def _patch(name, fn):
    return lambda mp, c, t: mp.setattr(O, name, fn(getattr(O, name)))


def _config(edit):
    return lambda mp, c, t: edit(c)


MISTAKES = {
    "no first row": _patch("bigram_rows", lambda f: lambda t, b, p, c: [c * t[0] % b] + f(t, b, p, c)[1:]),
    "bigram the other way round": _patch("bigram_rows", lambda f: lambda t, b, p, c: f(t, b, c, p)),
    "norm weight not around one": _patch("rms_around_one", lambda f: lambda x, w, eps: O.rms(x, eps) * w),
    "eps": _config(lambda c: c["norm"].update(eps=c["norm"]["eps"] * 3)),
    "halves turned": _patch("rotate_pairs", lambda f: lambda x, d, b: f(x[..., [0, 3, 1, 4, 2, 5, 6, 7, 8, 9]], d, b)),
    "a position late after 40 tokens": _patch("rotate_pairs", lambda f: lambda x, d, b: torch.cat([f(x, d, b)[:40], f(torch.cat([x[:1], x]), d, b)[41:]])),
    "scale": _config(lambda c: c["layers"][1]["mixer"]["left"].update(scale=c["layers"][1]["mixer"]["left"]["scale"] * 1.02)),
    "scales of the two sides": _config(lambda c: c["layers"][1]["mixer"].update(left_scale=1.0, right_scale=0.5)),
    "a tap less": _patch("short_conv", lambda f: lambda x, w: f(x, torch.cat([torch.zeros_like(w[:, :1]), w[:, 1:]], 1))),
    "taps turned round": _patch("short_conv", lambda f: lambda x, w: f(x, w.flip(1))),
    "no unit vectors": _patch("unit", lambda f: lambda x: x),
    "plain relu": _patch("relu_squared", lambda f: lambda z: z.clamp_min(0)),
    "no softplus": _patch("softplus", lambda f: torch.exp),
    "read before write": _patch("delta_rule", lambda f: lambda q, k, v, g, b: f(q, k, v, g, b) - _own_write(q, k, v, g, b)),
    "decay after the write": _patch("delta_rule", lambda f: lambda q, k, v, g, b: f(q, k, v, torch.cat([torch.ones_like(g[:1]), g[:-1]]), b)),
}  # fmt: skip


def _own_write(q, k, v, g, b):
    """The part of every output that the token's own write contributes: (k . q) u."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = b[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out.append((k[t] @ q[t]) * u)
    return torch.stack(out)


@pytest.mark.parametrize("mistake", sorted(MISTAKES) + ["no sink", "value heads", "decay channels", "gate"])
def test_a_mistake_in_the_definition_shows(mistake, monkeypatch):
    """The comparison is sharp: with one thing wrong in the definition the engine no longer agrees with it."""
    config = copy.deepcopy(O.CONFIGS["odd"])
    tensors, tokens = O.random_tensors(config, seed=1), O.random_tokens(config, 60, seed=1)
    got = feed_all(make_engine(config, tensors), [31, 2], tokens)
    assert O.error(got, O.forward(config, tensors, tokens)) < TOL
    if mistake == "no sink":
        soft = torch.softmax
        monkeypatch.setattr(torch, "softmax", lambda x, d: torch.cat([soft(x[:, :-1], d), x[:, -1:]], 1))
    elif mistake == "value heads":
        tensors = dict(tensors, **{"l0.mix.v": tensors["l0.mix.v"].roll(14, 0)})
    elif mistake == "decay channels":
        tensors = dict(tensors, **{"l1.mix.right.dt_bias": tensors["l1.mix.right.dt_bias"].roll(1, 0)})
    elif mistake == "gate":
        sigmoid = torch.sigmoid
        monkeypatch.setattr(O, "silu", lambda z: z * sigmoid(1.5 * z))
    else:
        MISTAKES[mistake](monkeypatch, config, tensors)
    assert O.error(got, O.forward(config, tensors, tokens)) > 5 * TOL


# ------------------------------------------------------------------------------------ configuration, loading, cache
def test_configuration_round_trip():
    for config in O.CONFIGS.values():
        tensors = O.random_tensors(config)
        cfg = ModelConfig.from_hf(config, O.shapes(tensors))
        assert cfg.num_params() == sum(v.numel() for v in tensors.values())
        written = json.loads(json.dumps(cfg.to_hf_dict()))
        assert ModelConfig.from_hf(written) == cfg  # carries the inner widths
        for layer in written["layers"]:
            for key in ("decay_rank", "gate_rank"):
                layer["mixer"].get("right", {}).pop(key, None)
        assert written == config
        assert [LayerSpec.of(s.to_dict()) for s in cfg.layer_specs] == cfg.layer_specs
    with pytest.raises(ValueError, match="inner width"):
        ModelConfig.from_hf(O.CONFIGS["single"])
    bad = copy.deepcopy(O.CONFIGS["rules"])
    bad["layers"][0]["type"] = "attention"
    with pytest.raises(ValueError, match="mixer"):
        ModelConfig.from_hf(bad)
    with pytest.raises(ValueError, match="layer_specs"):
        ModelConfig(num_layers=1, hidden_size=8, num_attention_heads=1, num_query_groups=1, ffn_hidden_size=8, vocab_size=8, norm_offset=1.0)


def test_loader_refuses_what_the_model_does_not_have():
    config = O.CONFIGS["mixed"]
    e = make_engine(config, O.random_tensors(config))
    z = torch.zeros(96, 96)
    for name in ("l0.norm2", "l1.mlp.up", "l0.mix.q", "l1.mix.a1", "l1.mix.left.q", "l0.mlp.gate", "l0.mix.right.g", "l4.norm1", "x"):
        assert e.update_weights([(name, z)]) == [name]
    with pytest.raises(ValueError, match="shape"):
        e.update_weights([("l0.mix.left.o", z)])
    assert set(e.weights.specified_tensors()) == set(O.random_tensors(config))


def test_recurrent_layers_behind_a_norm_of_their_own():
    """The parts serve other designs too: a sequential layer (mixer, then feed-forward) with a recurrent mixer, full-rank decay
    per channel beside a two-factor gate, fp8 asked for where only attention could use it."""
    from slime_b200.models.layer_spec import FeedForwardSpec, flat_sizes

    spec = LayerSpec(DeltaSpec(2, 1, 8, 12, 3, "channel", "silu", None, 6), FeedForwardSpec(20, "silu"))
    cfg = ModelConfig(**dict(flat_sizes([spec]), layer_specs=[spec], hidden_size=16, vocab_size=30, model_arch="Other", tie_word_embeddings=False))
    e = Engine(cfg, ServerArgs(page_size=8, max_running_requests=2, context_length=64), device="cpu", num_pages=17)
    names = e.weights.specified_tensors()
    assert names["l0.mix.a"] == (16, 16) and names["l0.mix.g1"] == (6, 16) and names["l0.mix.g2"] == (24, 6) and "l0.norm2" in names
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(*s, generator=g) * 0.4 for n, s in names.items()}
    assert not e.update_weights(t.items())
    tokens = O.random_tokens(dict(vocab=30), 30)
    x = t["embed"][tokens]
    W = lambda n: t["l0.mix." + n]  # noqa: E731
    h = O.rms(x, 1e-6) * t["l0.norm1"]
    y = O.short_conv(torch.cat([h @ W(n).t() for n in "qkv"], 1), torch.cat([W(n + ".conv") for n in "qkv"]))
    q, k, v = O.unit(y[:, :8]) * 8**-0.5, O.unit(y[:, 8:16]), y[:, 16:].view(-1, 2, 12)
    decay = torch.exp(-torch.exp(W("A_log"))[None, :, None] * O.softplus(h @ W("a").t() + W("dt_bias")).view(-1, 2, 8))
    o = torch.stack([O.delta_rule(q, k, v[:, i], decay[:, i], torch.sigmoid(h @ W("b").t())[:, i]) for i in range(2)], 1)
    x = x + ((O.rms(o, 1e-6) * W("norm")).flatten(1) * O.silu(h @ W("g1").t() @ W("g2").t())) @ W("o").t()
    h = O.rms(x, 1e-6) * t["l0.norm2"]
    x = x + (O.silu(h @ t["l0.mlp.gate"].t()) * (h @ t["l0.mlp.up"].t())) @ t["l0.mlp.down"].t()
    want = (O.rms(x, 1e-6) * t["final.norm"]) @ t["head"].t()
    assert cfg.norm_epsilon == 1e-6 and O.error(feed_all(e, [11, 2], tokens), want) < TOL


def test_what_a_recurrent_model_cannot_do_is_refused():
    from slime_b200.models.gpt import GPTModel

    config = O.CONFIGS["single"]
    tensors = O.random_tensors(config)
    with pytest.raises(NotImplementedError, match="rollout engine only"):
        GPTModel(ModelConfig.from_hf(config, O.shapes(tensors)), dtype=torch.float32, device="cpu")
    e = make_engine(config, tensors)
    with pytest.raises(NotImplementedError, match="recurrent state"):
        e.import_request([1, 2], 3, 0.0, (torch.zeros(1), torch.zeros(1)), dict(max_new_tokens=2))
    with pytest.raises(NotImplementedError, match="recurrent state"):
        e.export_kv(e.open_stream("a"))


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
    assert not (tmp_path / "1.f32").exists() and not r.live and len(r.engine.free_slots) == len(r.engine.states.free) == 4
    del tensors["l0.mix.right.q.conv"]
    save_file(tensors, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="missing"):
        trace.load_engine(str(tmp_path), "float32", 128, 64, 4, torch.device("cpu"))


def _rank_main(rank, port, config, tensors, tokens, want):
    import torch.distributed as dist

    torch.set_num_threads(1)
    dist.init_process_group("gloo", init_method=f"tcp://127.0.0.1:{port}", rank=rank, world_size=2)
    e = Engine(ModelConfig.from_hf(config, O.shapes(tensors)), ServerArgs(page_size=16, max_running_requests=4, context_length=128), device="cpu",
               num_pages=16, tp_group=dist.group.WORLD, tp_size=2, tp_rank=rank)  # fmt: skip
    assert not e.update_weights(tensors.items())
    assert O.error(feed_all(e, [17, 2, 20], tokens), want) < TOL
    dist.destroy_process_group()


def test_two_tensor_parallel_ranks():
    import socket

    config = O.model(48, 70, (29, 3, 7), [(O.both(O.attn(4, 2, 16, 24, 12), O.rule(6, 2, 12, 20, 4)), 40), (O.rule(4, 4, 8, 16, 3), None)])
    tensors, tokens = O.random_tensors(config, seed=3), O.random_tokens(config, 44, seed=3)
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    want = O.forward(config, tensors, tokens)
    torch.multiprocessing.spawn(_rank_main, args=(port, config, tensors, tokens, want), nprocs=2)
    with pytest.raises(ValueError, match="divide"):
        t = O.random_tensors(O.CONFIGS["odd"])
        Engine(ModelConfig.from_hf(O.CONFIGS["odd"], O.shapes(t)), ServerArgs(), device="cpu", num_pages=4, tp_size=2)

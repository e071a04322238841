"""Pebodra models in the engine against the plain definition (``pebodra_oracle``), fp32 on the CPU."""

import copy
import json

import pebodra_oracle as O
import pytest
import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.projections import LayerProjections
from slime_b200.engine.server_args import ServerArgs
from slime_b200.engine.state_cache import RecurrentStates, StateShape
from slime_b200.models.config import ModelConfig, get_preset
from slime_b200.models.layer_spec import AttentionSpec, FeedForwardSpec, LayerSpec, MatrixMemorySpec, ParallelSpec, StateSpaceSpec
from slime_b200.ops import grouped, linear_scan, stream
from slime_b200.ops import window_attention as wa

TOL = 1e-4


def make_engine(config, tensors, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, **kw}
    e = Engine(ModelConfig.from_hf(config), ServerArgs(page_size=page_size, **kw), device="cpu", num_pages=num_pages)
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
@pytest.mark.parametrize("groups", [1, 3, 6, 24])
def test_norms_of_parts_around_the_stream(groups):
    g = torch.Generator().manual_seed(0)
    y, res, w, pre = (torch.randn(*s, generator=g) for s in ((5, 24), (5, 24), (24,), (24,)))
    want = res + O.rms_parts(y, groups, 0.01) * w
    h, got = stream.stream_norm(y, res.clone(), pre, 0.01, post_w=w, groups=groups)
    torch.testing.assert_close(got, want)
    torch.testing.assert_close(h, O.rms_parts(want, groups, 0.01) * pre)
    h, got = stream.stream_norm(y, res.clone(), None, 0.01, post_w=w, groups=groups, emit=torch.bfloat16)
    assert torch.equal(h, got.bfloat16()) and stream.stream_norm(y, res.clone(), None, 0.01, post_w=w, groups=groups)[0] is None


def test_normed_polynomial():
    g = torch.Generator().manual_seed(1)
    z, coef = torch.randn(7, 30, generator=g) * 3, torch.randn(4, generator=g)
    want = O.poly_norm(z, coef, 0.01)
    torch.testing.assert_close(stream.poly_norm(z, coef, 0.01), want)
    sums = stream.poly_sums(z)  # two ranks have half of a row each
    halves = [stream.poly_norm(x, coef, 0.01, sums, 30) for x in z.split([12, 18], 1)]
    torch.testing.assert_close(torch.cat(halves, 1), want)
    x = torch.randn(3, 9, generator=g) * 30
    torch.testing.assert_close(stream.softcap_(x.clone(), 7.0), 7.0 * torch.tanh(x / 7.0))


@pytest.mark.parametrize("experts,top,groups", [(8, 3, (4, 2)), (6, 2, (6, 3)), (9, 2, (3, 1)), (7, 7, (1, 1)), (12, 4, (2, 2)), (1, 1, (1, 1))])
def test_router_prefers_good_groups(experts, top, groups):
    z = torch.randn(60, experts, generator=torch.Generator().manual_seed(top))
    w, idx = grouped.route_topk(z, top, score="sigmoid", renorm=False, groups=groups)
    s = torch.sigmoid(z)
    for t in range(60):
        assert idx[t].tolist() == O.choose(s[t], top, dict(count=groups[0], keep=groups[1]))
    torch.testing.assert_close(w, s.gather(1, idx))


def _pages(lengths, ps, *tensors):
    g = torch.Generator().manual_seed(len(lengths))
    count = [-(-n // ps) for n in lengths]
    order = torch.randperm(sum(count) + 2, generator=g).tolist()
    pages = [[order.pop() for _ in range(c)] for c in count]
    caches = []
    for per in tensors:
        c = torch.full(((sum(count) + 2) * ps, *per[0].shape[1:]), float("nan"))
        for p, rows in zip(pages, per):
            i = torch.arange(len(rows))
            c[torch.tensor(p)[i // ps] * ps + i % ps] = rows
        caches.append(c)
    return pages, caches


@pytest.mark.parametrize("window", [1, 7, 16, 200])
@pytest.mark.parametrize("ps", [4, 16])
def test_difference_of_two_attentions(window, ps):
    H, G, D, DV, lengths, starts = 6, 2, 6, 10, [70, 33, 1], [0, 31, 0]
    g = torch.Generator().manual_seed(ps)
    q, k, v = ([torch.randn(n, *s, generator=g) for n in lengths] for s in ((H, 2, D), (G, 2, D), (G, DV)))
    weight, gain, eps = torch.tensor([0.37]), 0.6, 0.01
    want = [O.pair_attention(*x, 0.9, O.window_mask(n, window), weight[0], 1 - gain, eps) for *x, n in zip(q, k, v, lengths)]
    pages, (kc, vc) = _pages(lengths, ps, [x.flatten(2) for x in k], v)
    batch = wa.ExtendBatch.build(pages, starts, [n - s for n, s in zip(lengths, starts)], ps, "cpu")
    wide = [torch.zeros(n, H, 2, 2, D) for n in lengths]  # each query beside zeros where the other key stands
    for x, w in zip(q, wide):
        w[:, :, 0, 0], w[:, :, 1, 1] = x[:, :, 0], x[:, :, 1]
    pair = wa.Pair(weight, gain, eps)
    rows = torch.cat([w[s:] for w, s in zip(wide, starts)]).view(-1, 2 * H, 2 * D)
    got = wa.window_extend(rows, kc, vc, batch, 0.9, window, pair=pair)
    torch.testing.assert_close(got, torch.cat([x[s:] for x, s in zip(want, starts)]), atol=1e-5, rtol=1e-5)
    for t in (0, 1, 6, 7, 8, 15, 16, 17, 69):  # first tokens, window and page borders
        one = torch.tensor([t], dtype=torch.int32)
        got = wa.window_decode(wide[0][t : t + 1].view(1, 2 * H, 2 * D), kc, vc, batch.block_table[:1], one + 1, one, ps, 0.9, window, pair=pair)
        torch.testing.assert_close(got[0], want[0][t], atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("own", [True, False])
def test_pairs_of_heads_are_placed(own):
    H, G, D, DV, T = 3, 3, 10, 7, 20
    g = torch.Generator().manual_seed(1)
    x, wq, wk = torch.randn(T, (H + G) * 2 * D + G * DV, generator=g), torch.randn(D, generator=g), torch.randn(D, generator=g)
    q, k, v = x.split([H * 2 * D, G * 2 * D, G * DV], 1)
    want_q = O.rotate_halves(O.rms_parts(q.reshape(T, 2 * H, D), 1, 0.01) * wq, 6, 30.0)
    want_k = O.rotate_halves(O.rms_parts(k.reshape(T, 2 * G, D), 1, 0.01) * wk, 6, 30.0)
    kc, vc = torch.full((32, G, 2 * D), 7.0), torch.full((32, G, DV), 7.0)
    slots = torch.arange(T, dtype=torch.int32)
    got = stream.place_heads(q, k if own else None, v if own else None, slots, kc, vc, q_norm=wq, k_norm=wk if own else None, eps=0.01,
                             table=stream.rotary_table(T, 6, 30.0), positions=slots, interleaved=False, maps=2)  # fmt: skip
    got = got.view(T, H, 2, 2, D)
    torch.testing.assert_close(torch.stack([got[:, :, 0, 0], got[:, :, 1, 1]], 2).flatten(1, 2), want_q, atol=1e-5, rtol=1e-5)
    assert not got[:, :, 0, 1].any() and not got[:, :, 1, 0].any()
    if own:
        torch.testing.assert_close(kc[:T].reshape(T, 2 * G, D), want_k, atol=1e-5, rtol=1e-5)
        assert torch.equal(vc[:T].flatten(1), v)
    else:
        assert (kc == 7).all() and (vc == 7).all()


def _ssm_mixer(shape, T, seed):
    H, G, N, DV, taps, parts = shape
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    widths = [H * DV, H * DV, G * N, G * N, H]
    cols = r(T, sum(widths)).split(widths, 1)
    ch = H * DV + 2 * G * N
    return linear_scan.StateSpace(*cols, r(ch, taps) * 0.6, r(ch) * 0.3, r(H) - 1, r(H) - 2, r(H), r(H * DV), parts, 0.01)


def _cut(x, lo, hi, names):
    import dataclasses

    return dataclasses.replace(x, **{n: getattr(x, n)[lo:hi] for n in names})


def _in_portions(mixer, names, state, cuts, T):
    out, at = [], 0
    for n in cuts:
        part = _cut(mixer, at, at + n, names)
        if n == 1:
            one = torch.ones(1, dtype=torch.int32)
            out.append(part.step(state, one, one, one * at))
        else:
            out.append(part.extend(state, wa.ExtendBatch.build([[0]], [at], [n], 256, "cpu", state_slots=[1])))
        at += n
    assert at == T
    return torch.cat(out)


CUTS = [[40], [1] * 40, [2] * 20, [7, 1, 1, 20, 2, 9], [3, 37]]


@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("shape", [(6, 2, 8, 5, 4, 3), (2, 1, 5, 12, 1, 1), (3, 3, 16, 4, 7, 2)])
def test_state_space(shape, cuts):
    H, G, N, DV, taps, parts = shape
    T, x = 40, _ssm_mixer(shape, 40, sum(shape))
    xBC = O.short_conv(torch.cat([x.x, x.B, x.C], 1), x.conv, x.conv_b).split([H * DV, G * N, G * N], 1)
    y = O.state_space(xBC[0].reshape(T, H, DV), xBC[1].reshape(T, G, N), xBC[2].reshape(T, G, N), torch.nn.functional.softplus(x.dt + x.dt_bias),
                      x.A_log.exp(), x.skip)  # fmt: skip
    want = O.rms_parts(y.reshape(T, -1) * O.silu(x.z), parts, 0.01) * x.norm
    state = linear_scan.SlotState(torch.full((3, H, N, DV), 7.0), torch.full((3, taps, H * DV + 2 * G * N), 7.0))  # whatever a slot held
    got = _in_portions(x, ("z", "x", "B", "C", "dt"), state, cuts, T)
    torch.testing.assert_close(got, want, atol=1e-4, rtol=1e-4)
    assert (state.state[[0, 2]] == 7).all() and (state.ring[[0, 2]] == 7).all()


@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("shape,bias", [((3, 8, 5), (0.0, 3.0)), ((1, 4, 12), (6.0, -4.0)), ((2, 6, 6), (-9.0, 9.0))])
def test_matrix_memory(shape, bias, cuts):
    """Gates around their caps: inputs that take over, a running maximum that only falls, a divisor at its least."""
    H, D, DV = shape
    T, g = 40, torch.Generator().manual_seed(D)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x = linear_scan.MatrixMemory(r(T, H * D), r(T, H * D), r(T, H * DV), 3 * r(T, H), 3 * r(T, H), r(T, H * DV), r(H) + bias[0], r(H) + bias[1],
                                 r(H * DV), 10.0, 0.01)  # fmt: skip
    soft = lambda z: 10.0 * torch.tanh(z / 10.0)  # noqa: E731
    y = O.matrix_memory(x.q.view(T, H, D) * D**-0.5, x.k.view(T, H, D), x.v.view(T, H, DV), soft(x.i + x.i_b), O.log_sigmoid(soft(x.f + x.f_b)))
    want = O.rms_parts(y, 1, 0.01).reshape(T, -1) * x.norm * torch.sigmoid(x.z)
    state = linear_scan.SlotState(torch.full((3, H, D, DV), 7.0), None, torch.full((3, H, D), 7.0), torch.full((3, H, 2), 7.0))
    got = _in_portions(x, "qkvzif", state, cuts, T)
    torch.testing.assert_close(got, want, atol=1e-4, rtol=1e-4)
    assert all((t[[0, 2]] == 7).all() for t in (state.state, state.norm, state.top))


def test_state_shapes():
    s = RecurrentStates([StateShape(2, 3, 4, 20, 4), StateShape(1, 8, 5, normalised=True)], 2, torch.bfloat16, torch.device("cpu"))
    assert s.of[0].ring.shape == (2, 4, 20) and s.of[0].ring.dtype == torch.bfloat16 and s.of[0].norm is None and s.of[0].top is None
    assert s.of[1].ring is None and s.of[1].norm.shape == (2, 1, 8) and s.of[1].top.shape == (2, 1, 2) and s.of[1].state.dtype == torch.float32
    assert s.num_bytes() == 4 * (2 * 24 + 2 * 40 + 16 + 4) + 2 * 2 * 80
    s.release()
    assert not s.of and not s.state
    s.allocate()
    assert len(s.of) == 2


def test_fused_matrices_hold_every_tensor_once():
    for config in O.CONFIGS.values():
        tensors = O.random_tensors(config)
        for i, spec in enumerate(ModelConfig.from_hf(config).layer_specs):
            lay = LayerProjections(spec)
            for ranges, total in ((lay.ins, lay.in_rows), (lay.outs, lay.out_cols)):
                at = 0
                for a, n in sorted(ranges.values()):
                    assert a >= at and a % 8 == 0
                    at = a + n
                assert at <= total
            shapes = lay.tensors(config["width"])
            assert shapes == {k[len(f"l{i}.") :]: tuple(v.shape) for k, v in tensors.items() if k.startswith(f"l{i}.mix.")}


# ------------------------------------------------------------------------------------ whole models
def test_prompt_portions_and_decoding_agree_with_the_definition(case):
    config, tensors, tokens, want = case
    n = len(tokens)
    for ps in (4, 16):
        e = make_engine(config, tensors, page_size=ps)
        for cuts in ([n], [n - 9], [1], [2] * 30, [3, 16, 29, 2, 2], [64], [37, 5]):
            err = O.error(feed_all(e, cuts, tokens), want)
            assert err < TOL, (ps, cuts, err)


def test_streams_of_every_layer(case):
    config, tensors, tokens, _ = case
    layers, got = [], []
    O.forward(config, tensors, tokens, layers_out=layers)
    e = make_engine(config, tensors)
    e.runner.stream_hook = lambda i, x: got.append(x.clone())
    feed_all(e, [len(tokens)], tokens)
    assert len(got) == len(layers)
    for a, b in zip(got, layers):
        torch.testing.assert_close(a, b.float(), atol=1e-3, rtol=1e-3)


def test_unequal_batches_equal_each_request_alone(case):
    config, tensors, _, _ = case
    e = make_engine(config, tensors, num_pages=1 + 4 * 4, page_size=16)  # four streams of 64 tokens: pages and slots are used again
    lengths = [64, 1, 40, 23, 64, 17, 2, 31]
    want = {i: O.forward(config, tensors, O.random_tokens(config, n, seed=i)) for i, n in enumerate(lengths)}
    g = torch.Generator().manual_seed(1)
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
            entries.append((req, O.random_tokens(config, lengths[i], seed=i)[at : at + n], list(range(n))))
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
    sp = [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps]
    reqs = e.generate(prompts, sp)
    for p, n, r in zip(prompts, steps, reqs):
        assert len(r.output_ids) == n
        picks = O.forward(config, tensors, p + r.output_ids).log_softmax(-1)[len(p) - 1 : -1]
        assert torch.equal(picks.argmax(-1), torch.tensor(r.output_ids))
        want = picks.gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
        assert float((want - torch.tensor(r.output_logprobs)).abs().max()) < 1e-3
    again = e.generate(prompts, sp)  # in used slots and pages
    assert [r.output_ids for r in again] == [r.output_ids for r in reqs] and len(e.states.free) == 3


def test_generation_under_page_pressure(case):
    config, tensors, _, _ = case
    prompts = [O.random_tokens(config, 30, seed=40 + i) for i in range(3)]
    sp = [dict(max_new_tokens=40, temperature=0, ignore_eos=True)] * 3
    roomy = make_engine(config, tensors, num_pages=64, page_size=8).generate(prompts, sp)
    tight = make_engine(config, tensors, num_pages=1 + 16, page_size=8)  # 128 tokens for 3 x 70: requests are retracted
    assert [r.output_ids for r in tight.generate(prompts, sp)] == [r.output_ids for r in roomy]


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding(name):
    config = O.CONFIGS[name]
    tensors, tokens = O.random_tensors(config, seed=2), O.random_tokens(config, 220, seed=3)
    assert O.error(feed_all(make_engine(config, tensors), [9], tokens), O.forward(config, tensors, tokens)) < TOL


def _marked(window, second=None):
    """Attention in which token 38 is a key that the query of token 39 matches and nothing else does, in the first of the two attentions;
    ``second``: a layer that uses its keys and values under a window of its own."""
    layers = [(O.attn(4, 2, 16, 12, window, 8, 100.0, scale=4.0), None)]
    if second:
        layers.append((O.attn(4, 2, 16, 12, second, 8, 100.0, scale=4.0, kv_from=0), None))
    config = O.model(48, 40, layers)
    t = O.random_tensors(config, seed=3, sharp=1.0)
    t["embed"][:, :2] = 0.0
    t["embed"][38, 0] = t["embed"][39, 1] = 40.0
    for i in range(len(layers)):
        for mark, x in enumerate("kq"):
            if f"l{i}.mix.{x}" not in t:
                continue
            w = t[f"l{i}.mix.{x}"].view(-1, 2, 16, 48)
            w.mul_(0.05)
            w[..., :2] = 0.0
            w[:, 0, 12, mark] = 20.0  # a coordinate that is not turned
            t[f"l{i}.mix.{x}.norm"][:] = 1.0
            t[f"l{i}.mix.{x}.b"].mul_(0.05)
        t[f"l{i}.norm1"].view(-1)[:2] = 0.0  # the marks stay
    return config, t


@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("size", [2, 7, 16, 33, 64])
def test_edges_of_windows(size, shared):
    """A matching key just inside the query's window decides, one just outside must not, in prompts and in decoding; the same where the
    window is that of a layer with another layer's keys."""
    config, tensors = _marked(1, size) if shared else _marked(size)
    for q in (size, 70):
        for back, inside in ((size - 1, True), (size, False)):
            tokens = [x % 38 for x in O.random_tokens(config, q + 1, seed=1)]
            tokens[q - back], tokens[q] = 38, 39
            want, other = O.forward(config, tensors, tokens), list(tokens)
            other[q - back] = 5
            moved = O.error(O.forward(config, tensors, other)[-1:], want[-1:])
            assert moved > 0.05 if inside else moved < 1e-12
            for ps in (4, 16):
                for cuts in ([q + 1], [q], [q - 1, 2]):
                    e = make_engine(config, tensors, page_size=ps, num_pages=512 // ps + 1)
                    assert O.error(feed_all(e, cuts, tokens), want) < TOL


@pytest.mark.parametrize("kind", ["mamba2", "mlstm"])
@pytest.mark.parametrize("cut", [0, 60])
def test_a_token_far_back_is_remembered(kind, cut):
    """With decays near one a token 140 positions back moves the answer, whether the prompt is one portion or the last tokens are decoded."""
    mixer = O.ssm(2, 1, 24, 16) if kind == "mamba2" else O.memory(2, 16, 16)
    config = O.model(48, 40, [(mixer, None)])
    t = O.random_tensors(config, seed=3)
    if kind == "mamba2":
        t["l0.mix.A_log"][:] = -8.0
        t["l0.mix.D"][:] = 0.0
    else:
        t["l0.mix.f.b"][:], t["l0.mix.i.b"][:] = 40.0, 0.0  # the cap bounds it: a forget gate of sigmoid(12)
    tokens = O.random_tokens(config, 150, seed=1)
    want, other = O.forward(config, t, tokens), list(tokens)
    other[9] = (other[9] + 1) % 40
    assert O.error(O.forward(config, t, other)[-1:], want[-1:]) > 20 * TOL
    e = make_engine(config, t)
    for cuts in ([150 - cut], [10, 1, 2, 137 - cut]):
        assert O.error(feed_all(e, cuts, tokens), want) < TOL


def _patch(name, fn):
    return lambda mp, c, t: mp.setattr(O, name, fn(getattr(O, name)))


def _edit(layer, part="mixer", **kw):
    return lambda mp, c, t: c["layers"][layer][part].update(kw)


def _tensor(name, fn):
    return lambda mp, c, t: t.update({name: fn(t[name])})


MISTAKES = {  # of the model "odd": attention, mamba2, mlstm, attention with the first one's keys
    "eps": lambda mp, c, t: c["norm"].update(eps=c["norm"]["eps"] * 3),
    "one norm for the row": lambda mp, c, t: c["norm"].update(groups=1),
    "cap of the logits": lambda mp, c, t: c.update(logit_softcap=3.2),
    "no cap of the logits": lambda mp, c, t: c.update(logit_softcap=None),
    "window": _edit(0, mask=dict(size=8)),
    "window of the shared keys": _edit(3, mask=dict(size=7)),
    "scale": _edit(0, scale=0.33),
    "diff": _edit(3, diff=0.69),
    "difference without the factor": _patch("pair_weight", lambda f: lambda *a: f(*a) * 0 + 1),
    "vectors' exponentials": _patch("pair_weight", lambda f: lambda a, b, c, d, diff: (a * b).sum() - (c * d).sum() + diff),
    "maps the other way": _patch("pair_attention", lambda f: lambda q, k, *a: f(q.flip(2), k.flip(2), *a)),
    "heads of map 1 first": _patch("pair_attention", lambda f: lambda q, k, *a: f(q.transpose(1, 2).reshape(q.shape), k, *a)),
    "pairs next to each other": _patch("rotate_halves", lambda f: lambda x, d, b: f(x[..., [0, 2, 4, 1, 3, 5] + list(range(6, x.shape[-1]))], d, b)[..., [0, 3, 1, 4, 2, 5] + list(range(6, x.shape[-1]))]),
    "a position late after 40 tokens": _patch("rotate_halves", lambda f: lambda x, *a: torch.cat([f(x, *a)[:40], f(torch.cat([x[:1], x]), *a)[41:]])),
    "no query bias": _tensor("l3.mix.q.b", torch.zeros_like),
    "no value bias": _tensor("l0.mix.v.b", torch.zeros_like),
    "no output bias": _tensor("l0.mix.o.b", torch.zeros_like),
    "key norm": _tensor("l0.mix.k.norm", lambda x: x.roll(1)),
    "softplus": _tensor("l1.mix.dt_bias", lambda x: x + 0.05),
    "decay": _tensor("l1.mix.A_log", lambda x: x + 0.05),
    "skip": _tensor("l1.mix.D", torch.zeros_like),
    "convolution backwards": _tensor("l1.mix.conv", lambda x: x.flip(1)),
    "no bias of the convolution": _tensor("l1.mix.conv.b", torch.zeros_like),
    "norm before the gate": _patch("rms_parts", lambda f: lambda x, p, e: f(x, 1 if p == 3 else p, e)),
    "norm of the heads as a whole": _edit(1, norm_groups=1),
    "no least divisor": _patch("matrix_memory", lambda f: lambda q, k, v, i, g: f(q, k, v, i + 30, g)),
    "cap of the gates": _edit(2, gate_cap=5.0),
    "query scale": _patch("matrix_memory", lambda f: lambda q, *a: f(q * 5**0.5, *a)),
    "input gate bias": _tensor("l2.mix.i.b", torch.zeros_like),
    "output gate": _tensor("l2.mix.g", lambda x: x.roll(1, 0)),
    "state lost after 31 tokens": _patch("state_space", lambda f: lambda x, B, C, s, *a: torch.cat([f(*(t[o] for t in (x, B, C, s)), *a) for o in (slice(0, 31), slice(31, None))])),
    "memory lost after 31 tokens": _patch("matrix_memory", lambda f: lambda *a: torch.cat([f(*(t[o] for t in a)) for o in (slice(0, 31), slice(31, None))])),
    "convolution starts anew": _patch("short_conv", lambda f: lambda x, w, b: torch.cat([f(x[:31], w, b), f(x[31:], w, b)])),
    "norms of the powers": _patch("poly_norm", lambda f: lambda z, c, e: sum(c[i] * O.rms_parts(z, 1, e) ** (i + 1) for i in range(3)) + c[3]),
    "no constant": _tensor("l0.mlp.act", lambda x: x * torch.tensor([1.0, 1.0, 1.0, 0.0])),
    "groups of experts": lambda mp, c, t: c["layers"][1]["mlp"]["router"].update(groups=dict(count=3, keep=2)),
    "group's best expert alone": _patch("choose", lambda f: lambda s, top, g: _by_best(s, top, g)),
    "weights over the chosen": _patch("experts", lambda f: lambda h, W, m: f(h, lambda n: W(n) * (0.9 if n.endswith("down") else 1.0), m)),
    "a norm in front": _patch("experts", lambda f: lambda h, W, m: f(O.rms_parts(h, 1, 1e-3), W, m)),
}  # fmt: skip


def _by_best(s, top, groups):
    per = s.shape[0] // groups["count"]
    kept = sorted(range(groups["count"]), key=lambda g: -float(s[g * per : (g + 1) * per].max()))[: groups["keep"]]
    return sorted([e for g in kept for e in range(g * per, (g + 1) * per)], key=lambda e: -float(s[e]))[:top]


@pytest.fixture(scope="module")
def odd():
    config = copy.deepcopy(O.CONFIGS["odd"])
    config["layers"][1]["mlp"] = O.moe(9, 2, 13, (3, 1))  # groups of three: their best expert alone is another choice
    tensors, tokens = O.random_tensors(config, seed=1), O.random_tokens(config, 60, seed=1)
    got = feed_all(make_engine(config, tensors), [31, 2], tokens)
    assert O.error(got, O.forward(config, tensors, tokens)) < TOL
    return config, tensors, tokens, got


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_in_the_definition_shows(mistake, odd, monkeypatch):
    """The comparison is sharp: with one thing wrong in the definition the engine no longer agrees with it."""
    config, tensors, tokens, got = odd
    config, tensors = copy.deepcopy(config), dict(tensors)
    MISTAKES[mistake](monkeypatch, config, tensors)
    assert O.error(got, O.forward(config, tensors, tokens)) > 5 * TOL


# ------------------------------------------------------------------------------------ configuration, loading, cache
def test_configuration_round_trip():
    for config in O.CONFIGS.values():
        cfg = ModelConfig.from_hf(config)
        assert cfg.num_params() == sum(v.numel() for v in O.random_tensors(config).values())
        written = json.loads(json.dumps(cfg.to_hf_dict()))
        assert written == config and ModelConfig.from_hf(written) == cfg
        assert [LayerSpec.of(s.to_dict()) for s in cfg.layer_specs] == cfg.layer_specs
    bad = copy.deepcopy(O.CONFIGS["single"])
    bad["layers"][1]["type"] = "delta"
    with pytest.raises(ValueError, match="mixer"):
        ModelConfig.from_hf(bad)
    bad = copy.deepcopy(O.CONFIGS["single"])
    bad["layers"][0]["mlp"]["kind"] = "gated"
    with pytest.raises(ValueError, match="feed-forward"):
        ModelConfig.from_hf(bad)
    for j, what in ((0, dict(heads=2)), (2, {}), (3, {}), (0, dict(rot=dict(dims=4, base=10.0)))):  # other geometry, no keys, itself
        bad = copy.deepcopy(O.CONFIGS["odd"])
        bad["layers"][3]["mixer"].update(kv_from=j, **what)
        if "heads" in what:
            bad["layers"][3]["mixer"].update(kv_heads=2)
        with pytest.raises(ValueError, match="keys and values of layer"):
            ModelConfig.from_hf(bad)
    for kw in (dict(logit_softcap=2.0), dict(norm_groups=2), dict(pre_norm=False)):
        with pytest.raises(ValueError, match="layer_specs"):
            ModelConfig(num_layers=1, hidden_size=8, num_attention_heads=1, num_query_groups=1, ffn_hidden_size=8, vocab_size=8, **kw)
    optional = copy.deepcopy(O.CONFIGS["single"])  # groups of experts, and of the norm, may be left out
    del optional["layers"][0]["mlp"]["router"]["groups"], optional["norm"]["groups"]
    assert ModelConfig.from_hf(optional) == ModelConfig.from_hf(O.CONFIGS["single"])


def test_mechanism_parameters_that_do_not_fit_are_refused():
    for kw in (dict(diff=0.5, sink=0.0), dict(diff=0.5, gate="head"), dict(diff=0.5, distance_bias="geometric"), dict(kv_from=-1),
               dict(diff=0.5, qk_norm=True, norm_over="projection")):  # fmt: skip
        with pytest.raises(ValueError):
            AttentionSpec(4, 2, 8, 16, 1.0, **kw)
    for spec, args in ((StateSpaceSpec, (3, 2, 8, 8, 4)), (StateSpaceSpec, (2, 1, 8, 8, 0)), (StateSpaceSpec, (2, 1, 8, 8, 4, 3)), (MatrixMemorySpec, (2, 8, 8, 0.0))):
        with pytest.raises(ValueError):
            spec(*args)
    for kw in (dict(expert_groups=3, keep_groups=1), dict(expert_groups=4, keep_groups=1), dict(expert_groups=2, keep_groups=3), dict(score="tanh")):
        with pytest.raises(ValueError):
            FeedForwardSpec(8, "silu", experts=8, top=3, **{"score": "sigmoid", **kw})
    for kw in (dict(), dict(gated=False, experts=2)):
        with pytest.raises(ValueError, match="polynomial"):
            FeedForwardSpec(8, "poly_norm", **kw)
    with pytest.raises(ValueError, match="side by side"):
        ParallelSpec(AttentionSpec(2, 1, 8, 8, 1.0, kv_from=0), MatrixMemorySpec(2, 8, 8, 5.0))


def test_loader_refuses_what_the_model_does_not_have():
    config = O.CONFIGS["mixed"]
    e = make_engine(config, O.random_tensors(config))
    z = torch.zeros(96, 96)
    for name in ("l2.norm2", "l0.norm1b", "l0.mix.q", "l3.mix.k", "l3.mix.v.b", "l3.mix.k.norm", "l0.mix.z", "l0.mix.in.b", "l2.mix.q.b", "l2.mix.conv",
                 "l1.mlp.e8.up", "l0.mlp.gate", "l1.mlp.act", "embed.norm", "l9.norm1", "x"):  # fmt: skip
        assert e.update_weights([(name, z)]) == [name]
    with pytest.raises(ValueError, match="shape"):
        e.update_weights([("l0.mix.in", z)])
    assert set(e.weights.specified_tensors()) == set(O.random_tensors(config))
    assert e.kv.num_layers == 2 and len(e.states.of) == 4  # layers with another one's keys have no cache of their own


def test_weights_can_be_replaced():
    """A second load (a trainer's update) reaches everything that is derived from a tensor, the factor of a pair included."""
    config = O.CONFIGS["mixed"]
    tokens = O.random_tokens(config, 40, seed=1)
    e = make_engine(config, O.random_tensors(config, seed=1))
    feed_all(e, [30], tokens)
    second = O.random_tensors(config, seed=2)
    e.update_weights(second.items())
    assert O.error(feed_all(e, [30], tokens), O.forward(config, second, tokens)) < TOL


def test_presets():
    for name in ("pebodra-4b", "pebodra-a3b", "pebodra-tiny"):
        cfg = get_preset(name)
        assert cfg.model_arch == "Pebodra" and {type(s.mixer).__name__ for s in cfg.layer_specs} == {"AttentionSpec", "StateSpaceSpec", "MatrixMemorySpec"}
        assert ModelConfig.from_hf(cfg.to_hf_dict()) == cfg
    e = Engine(get_preset("pebodra-tiny"), ServerArgs(page_size=16, max_running_requests=2, context_length=128), device="cpu", num_pages=20)
    e.weights.init_random(0)
    assert len(e.generate([[1, 2, 3]], [dict(max_new_tokens=5, temperature=0, ignore_eos=True)])[0].output_ids) == 5


def test_the_parts_serve_other_designs():
    """Norms in front, a state space beside a matrix memory with factors, pairs without norms or biases, a gated dense feed-forward beside the
    mixer, routed experts with a bias and groups."""
    from slime_b200.models.layer_spec import RotarySpec, flat_sizes

    both = ParallelSpec(StateSpaceSpec(2, 1, 6, 8, 3, 2), MatrixMemorySpec(2, 6, 5, 7.0), 0.6, 1.4)
    pairs = AttentionSpec(4, 2, 6, 10, 0.5, window=9, rot=RotarySpec(4, 50.0), diff=0.2)
    specs = [LayerSpec(both, FeedForwardSpec(12, "silu"), parallel_ff=True),
             LayerSpec(pairs, FeedForwardSpec(12, "relu2", False, 6, 2, score="sigmoid", renorm=True, expert_groups=3, keep_groups=2))]  # fmt: skip
    cfg = ModelConfig(**dict(flat_sizes(specs), layer_specs=specs, hidden_size=16, vocab_size=30, model_arch="Other", tie_word_embeddings=False))
    e = Engine(cfg, ServerArgs(page_size=8, max_running_requests=2, context_length=64), device="cpu", num_pages=17)
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(*s, generator=g) * 0.5 for n, s in e.weights.specified_tensors().items()}
    assert not e.update_weights(t.items())
    tokens = O.random_tokens(dict(vocab=30), 40)
    T, eps = len(tokens), 1e-6
    norm = lambda x, n: O.rms_parts(x, 1, eps) * t[n]  # noqa: E731
    x = t["embed"][tokens]
    h = norm(x, "l0.norm1")
    part = lambda p: lambda n: t[f"l0.mix.{p}.{n}"]  # noqa: E731
    y = 0.6 * O.mamba2(h, part("left"), dict(heads=2, vdim=8, state=6, groups=1, norm_groups=2), eps)
    y = y + 1.4 * O.mlstm(h, part("right"), dict(heads=2, dim=6, gate_cap=7.0), eps)
    x = x + y + (O.silu(h @ t["l0.mlp.gate"].t()) * (h @ t["l0.mlp.up"].t())) @ t["l0.mlp.down"].t()
    h = norm(x, "l1.norm1")
    turn = lambda v: O.rotate_halves(v[..., [0, 2, 1, 3, 4, 5]], 4, 50.0)[..., [0, 2, 1, 3, 4, 5]]  # noqa: E731
    q, k, v = (h @ t[f"l1.mix.{n}"].t() for n in "qkv")
    q, k = turn(q.view(T, 8, 6)).view(T, 4, 2, 6), turn(k.view(T, 4, 6)).view(T, 2, 2, 6)
    lam = O.pair_weight(*(t["l1.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")), 0.2)
    x = x + O.pair_attention(q, k, v.view(T, 2, 10), 0.5, O.window_mask(T, 9), lam, 0.2, eps).reshape(T, -1) @ t["l1.mix.o"].t()
    h = norm(x, "l1.norm2")
    s = torch.sigmoid(h @ t["l1.mlp.router"].t())
    one = lambda j, z: torch.relu(z @ t[f"l1.mlp.e{j}.up"].t()) ** 2 @ t[f"l1.mlp.e{j}.down"].t()  # noqa: E731
    picks = [O.choose(s[i], 2, dict(count=3, keep=2)) for i in range(T)]
    x = x + torch.stack([sum(s[i, j] * one(j, h[i]) for j in c) / s[i, c].sum() for i, c in enumerate(picks)])
    want = norm(x, "final.norm") @ t["head"].t()
    assert O.error(feed_all(e, [11, 2], tokens), want) < TOL


def test_trainer_says_that_it_cannot_train_this():
    from slime_b200.models.gpt import GPTModel

    with pytest.raises(NotImplementedError, match="rollout engine only"):
        GPTModel(ModelConfig.from_hf(O.CONFIGS["single"]), dtype=torch.float32, device="cpu")


def test_attention_alone_uses_the_prefix_cache_and_travels():
    """Without recurrent layers prompts share pages, evicted pages come back from host memory, and keys travel between engines."""
    config = O.model(64, 90, [(O.attn(4, 2, 16, 24, 30, 8), O.moe(4, 2, 16, (2, 1))), (O.attn(4, 2, 16, 24, 12, 8, kv_from=0), O.plain(40))], norm_groups=2)
    tensors, prompt = O.random_tensors(config, seed=8), O.random_tokens(config, 45, seed=8)
    sp = dict(max_new_tokens=10, temperature=0, ignore_eos=True)
    a, b = make_engine(config, tensors), make_engine(config, tensors)
    want = a.generate([prompt], [sp])[0]
    picks = O.forward(config, tensors, prompt + want.output_ids)[len(prompt) - 1 : -1].argmax(-1)
    assert picks.tolist() == want.output_ids
    again = a.generate([prompt], [sp])[0]
    assert again.output_ids == want.output_ids and again.num_cached_tokens == 32
    pre = a.generate([prompt], [sp], prefill_only=True)[0]
    r = b.import_request(prompt, pre.output_ids[0], pre.output_logprobs[0], pre.kv_export, sp)
    while not r.finished():
        b.step()
    assert r.output_ids == want.output_ids
    small = make_engine(config, tensors, num_pages=9, enable_hierarchical_cache=True, hicache_ratio=4.0)
    small.generate([prompt], [sp])
    for i in range(3):
        small.generate([O.random_tokens(config, 60, seed=60 + i)], [sp])
    assert small.generate([prompt], [sp])[0].output_ids == want.output_ids and small.kv.allocator.host_tier.hits > 0


def test_replay_writes_the_wanted_logits(tmp_path):
    from safetensors.torch import save_file

    from slime_b200.engine import trace

    config = O.CONFIGS["mixed"]
    tensors = O.random_tensors(config, seed=4)
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_file(tensors, str(tmp_path / "model.safetensors"))
    r = trace.Replay(trace.load_engine(str(tmp_path), "float32", 128, 64, 4, torch.device("cpu")), str(tmp_path))
    a, b = O.random_tokens(config, 40, seed=1), O.random_tokens(config, 9, seed=2)
    r.step({"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [32, 0]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []})
    r.step({"step": 1, "entries": [{"id": "a", "tokens": a[33:34], "want": []}], "end": []})
    r.step({"step": 2, "entries": [{"id": "b", "tokens": b[1:], "want": [7]}, {"id": "a", "tokens": a[34:35], "want": [0]}], "end": ["a", "b"]})
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 203)  # noqa: E731
    la, lb = O.forward(config, tensors, a), O.forward(config, tensors, b)
    assert O.error(read(0), la[[32, 0]]) < TOL and O.error(read(2), torch.stack([lb[8], la[34]])) < TOL
    assert not (tmp_path / "1.f32").exists() and not r.live and len(r.engine.states.free) == 4
    for gone in ("l0.mix.in", "l1.mix.lq2", "l2.mix.f.b", "l1.mix.o.b", "l0.mlp.act", "head"):
        save_file({k: v for k, v in tensors.items() if k != gone}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ValueError, match="missing"):
            trace.load_engine(str(tmp_path), "float32", 128, 64, 4, torch.device("cpu"))


def _rank_main(rank, port, config, tensors, tokens, want, ep):
    import torch.distributed as dist

    torch.set_num_threads(1)
    dist.init_process_group("gloo", init_method=f"tcp://127.0.0.1:{port}", rank=rank, world_size=2)
    e = Engine(ModelConfig.from_hf(config), ServerArgs(page_size=16, max_running_requests=4, context_length=128, ep_size=ep), device="cpu", num_pages=16,
               tp_group=dist.group.WORLD, tp_size=2, tp_rank=rank)  # fmt: skip
    assert not e.update_weights(tensors.items())
    assert O.error(feed_all(e, [17, 2, 20], tokens), want) < TOL
    dist.destroy_process_group()


@pytest.mark.parametrize("ep", [1, 2])
def test_two_tensor_parallel_ranks(ep):
    import socket

    config = O.model(48, 70, [(O.ssm(4, 2, 8, 12, 3, 2), O.plain(40)), (O.attn(4, 2, 16, 12, 11, 8), O.moe(6, 3, 24, (3, 2))), (O.memory(2, 8, 12), O.moe(4, 1, 16)),
                              (O.attn(4, 2, 16, 12, 30, 8, kv_from=1), None)], norm_groups=3)  # fmt: skip
    tensors, tokens = O.random_tensors(config, seed=3), O.random_tokens(config, 44, seed=3)
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    want = O.forward(config, tensors, tokens)
    torch.multiprocessing.spawn(_rank_main, args=(port, config, tensors, tokens, want, ep), nprocs=2)
    for bad in (O.CONFIGS["odd"], O.model(48, 70, [(O.ssm(4, 2, 8, 12, 3, 1), None)])):
        with pytest.raises(ValueError, match="divide"):
            Engine(ModelConfig.from_hf(bad), ServerArgs(), device="cpu", num_pages=4, tp_size=2)

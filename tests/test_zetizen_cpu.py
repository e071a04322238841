"""Zetizen models in the engine against the plain definition (``zetizen_oracle``), fp32 on the CPU."""

import copy
import json
import math

import pytest
import torch
import zetizen_oracle as O

from slime_b200.engine.engine import Engine
from slime_b200.engine.projections import LayerProjections
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig, get_preset
from slime_b200.models.layer_spec import AttentionSpec, DistanceBiasSpec, FeedForwardSpec, LatentSpec, LayerSpec, RotarySpec, YarnSpec
from slime_b200.ops import grouped, latent, stream
from slime_b200.ops import window_attention as wa

TOL = 1e-4


def make_engine(model, tensors, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, **kw}
    e = Engine(ModelConfig.from_hf(model[0], O.shapes(tensors)), ServerArgs(page_size=page_size, **kw), device="cpu", num_pages=num_pages)
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


@pytest.fixture(scope="module", params=sorted(O.MODELS))
def case(request):
    model = O.MODELS[request.param]
    tensors = O.random_tensors(model, seed=5)
    tokens = O.random_tokens(model[0], 75, seed=6)
    return model, tensors, tokens, O.forward(model[0], tensors, tokens)


# ------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("rows,far", [(2, 3), (6, 17), (16, 64), (16, 100), (32, 128), (7, 50), (64, 1500)])
def test_distance_buckets(rows, far):
    spec = DistanceBiasSpec(rows, far)
    table = spec.by_distance()
    assert [spec.bucket(n) for n in range(2 * far)] == [O.bucket(n, rows, far) for n in range(2 * far)]
    assert table == [O.bucket(n, rows, far) for n in range(len(table))] and table[-1] == rows - 1 != table[-2]
    assert table[: rows // 2] == list(range(rows // 2)) and spec.bucket(far) == rows - 1
    for n in range(rows // 2, far):  # the bucket's number is the exact logarithm's floor
        b = spec.bucket(n) - rows // 2
        half = rows // 2
        assert (n / half) ** (rows - half) >= (far / half) ** b * (1 - 1e-9)
        assert b + half == rows - 1 or (n / half) ** (rows - half) < (far / half) ** (b + 1) * (1 + 1e-9)
    with pytest.raises(ValueError, match="buckets"):
        DistanceBiasSpec(rows, rows // 2)


@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, (4.0, 64, 8.0, 1.0)), (32, 2e4, (8.0, 2048, 32.0, 1.0)), (6, 50.0, (2.0, 32, 4.0, 0.5)),
                                               (4, 100.0, (1.0, 128, 32.0, 1.0)), (20, 5e5, None)])  # fmt: skip
def test_stretched_rotation(dims, base, scaling):
    names = ("factor", "original", "fast", "slow")
    rot = dict(dims=dims, base=base, scaling=dict(zip(names, scaling)) if scaling else None)
    spec = RotarySpec(dims, base, False, YarnSpec(*scaling) if scaling else None)
    freq, gain = O.yarn(dims, base, rot["scaling"])
    assert spec.frequencies() == pytest.approx(freq, rel=1e-14) and spec.gain() == pytest.approx(gain)
    if scaling and scaling[0] > 1:  # slow pairs are stretched, the fastest is not
        assert freq[-1] < base ** (-2 * (dims // 2 - 1) / dims) and gain > 1
    x = torch.randn(300, 2, dims + 6, dtype=torch.float64)
    table = stream.rotary_table(300, dims, base, frequencies=spec.frequencies(), gain=spec.gain())
    got = stream._turn(x.float(), table, torch.arange(300), False)
    torch.testing.assert_close(got.double(), O.rotate_halves(x, rot), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("tied", [False, True])
def test_heads_normed_over_the_whole_projection(tied):
    H, G, D, T, ps = 6, 3, 10, 41, 8
    g = torch.Generator().manual_seed(1)
    x, wq, wk = torch.randn(T, (H + 2 * G) * D, generator=g), torch.randn(H * D, generator=g), torch.randn(G * D, generator=g)
    q, k, v = x.split([H * D, G * D, G * D], 1)
    v = k if tied else v
    rot = O.yarn_rot(6, 30.0)
    spec = RotarySpec(6, 30.0, False, YarnSpec(**rot["scaling"]))
    table = stream.rotary_table(T, 6, 30.0, frequencies=spec.frequencies(), gain=spec.gain())
    kc, vc = torch.zeros(48, G, D), torch.zeros(48, G, D)
    before = k.clone()
    want_q, want_k = O.rms(q, wq, 0.01).view(T, H, D), O.rms(k, wk, 0.01).view(T, G, D)
    sums = (stream.head_sums(q, k), (H * D, G * D))
    half = stream.place_heads(q[:, : H * D // 2].clone(), k[:, : G * D], v, torch.full((T,), -1, dtype=torch.int32), kc, vc, q_norm=wq[: H * D // 2],
                              k_norm=wk, eps=0.01, sums=sums)  # fmt: skip
    torch.testing.assert_close(half, want_q[:, : H // 2])  # a part of the projection under the whole one's norm
    got = stream.place_heads(q, k, v, torch.arange(T, dtype=torch.int32), kc, vc, q_norm=wq, k_norm=wk, eps=0.01, table=table,
                             positions=torch.arange(T), interleaved=False)  # fmt: skip
    torch.testing.assert_close(got, O.rotate_halves(want_q, rot), atol=1e-5, rtol=1e-5)
    torch.testing.assert_close(kc[:T], O.rotate_halves(want_k, rot), atol=1e-5, rtol=1e-5)
    assert torch.equal(vc[:T].flatten(1), before if tied else v)


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


@pytest.mark.parametrize("form", ["bias", "chunk"])
@pytest.mark.parametrize("ps", [4, 16])
def test_scores_and_visibility(form, ps):
    H, G, D, DV, lengths, starts = 4, 2, 6, 10, [70, 33, 1], [0, 31, 0]
    g = torch.Generator().manual_seed(ps)
    q, k, v = ([torch.randn(n, h, w, generator=g) for n in lengths] for h, w in ((H, D), (G, D), (G, DV)))
    table, gate = torch.randn(10, H, generator=g) * 2, torch.randn(70 + 2 + 1, H, generator=g)
    kw = dict(softcap=2.0)
    bias = see = None
    if form == "bias":
        bias = O.distance_bias(table, 70, 40)
        kw["bias"] = table[DistanceBiasSpec(10, 40).by_distance()].contiguous()
    else:
        kw["chunk"] = 16
    see = [O.chunk_mask(n, 16) if form == "chunk" else O.causal(n) for n in lengths]
    want = [O.attend(*x, 0.9, s, 2.0, None if bias is None else bias[:, :n, :n]) for *x, s, n in zip(q, k, v, see, lengths)]
    pages, (kc, vc) = _pages(lengths, ps, k, v)
    counts = [n - s for n, s in zip(lengths, starts)]
    batch = wa.ExtendBatch.build(pages, starts, counts, ps, "cpu")
    rows = torch.cat([x[s:] for x, s in zip(want, starts)])
    got = wa.window_extend(torch.cat([x[s:] for x, s in zip(q, starts)]), kc, vc, batch, 0.9, gate=gate, **kw)
    torch.testing.assert_close(got, rows * torch.sigmoid(gate)[..., None], atol=1e-5, rtol=1e-5)
    for t in (0, 1, 15, 16, 17, 31, 32, 33, 69):  # first tokens, chunk and page borders
        one = torch.tensor([t], dtype=torch.int32)
        got = wa.window_decode(q[0][t : t + 1], kc, vc, batch.block_table[:1], one + 1, one, ps, 0.9, **kw)
        torch.testing.assert_close(got[0], want[0][t], atol=1e-5, rtol=1e-5)


def test_latent_attention_in_absorbed_form():
    H, D, r, DV, R, R1, T, ps = 3, 6, 4, 5, 11, 7, 40, 8
    g = torch.Generator().manual_seed(0)
    m = O.latent(H, D, r, DV, R1, R)
    shapes = dict(dq=(R1, 24), dkv=(R + r, 24), uq=(H * (D + r), R1), uk=(H * D, R), uv=(H * DV, R), g=(H * DV, 24), o=(24, H * DV))
    W = {n: torch.randn(*s, generator=g) * 0.4 for n, s in shapes.items()}
    W["dq.norm"], W["dkv.norm"] = torch.randn(R1, generator=g), torch.randn(R, generator=g)
    h = torch.randn(T, 24, generator=g)
    want = O.latent_attention(h, lambda n: W[n], m, 0.01)
    spec = RotarySpec(r, m["rot"]["base"], False, YarnSpec(**m["rot"]["scaling"]))
    table = stream.rotary_table(T, r, spec.base, frequencies=spec.frequencies(), gain=spec.gain())
    cache, pages = torch.zeros(6 * ps, 1, R + r), [5, 0, 3, 1, 4]
    slots = torch.tensor([pages[p // ps] * ps + p % ps for p in range(T)], dtype=torch.int32)
    batch = wa.ExtendBatch.build([pages], [0], [T], ps, "cpu")
    c = latent.latent_place(h @ W["dq"].t(), h @ W["dkv"].t(), W["dq.norm"], W["dkv.norm"], 0.01, table, batch.positions, slots, cache)
    q = (c @ W["uq"].t()).view(T, H, D + r)
    L = latent.Latent(H, D, DV, R, m["scale"], W["uq"], torch.cat([W["uk"], W["uv"]]), table)
    gate = (h @ W["g"].t()).view(T, H, DV)
    out = latent.latent_extend(L, q, cache, batch, gate, torch.empty(T, H, DV))
    torch.testing.assert_close(out.flatten(1) @ W["o"].t(), want, atol=1e-4, rtol=1e-4)
    for t in (0, 7, 8, 39):
        one = torch.tensor([t], dtype=torch.int32)
        out = latent.latent_decode(L, q[t : t + 1], cache, batch.block_table, one, ps, 64, gate[t : t + 1], torch.empty(1, H, DV))
        torch.testing.assert_close(out.flatten(1) @ W["o"].t(), want[t : t + 1], atol=1e-4, rtol=1e-4)


def test_expansion_tables_cover_the_long_requests():
    pages = [[7, 2, 9], [4], [1, 3], [5, 6, 8, 0]]
    b = wa.ExtendBatch.build(pages, [20, 0, 3, 0], [21, 2, 20, 64], 16, "cpu")
    ids, table, tiles = b.expansion((0, 3), 16)
    assert ids.tolist() == [7, 2, 9, 5, 6, 8, 0]
    assert table[0, :3].tolist() == [0, 1, 2] and table[3].tolist() == [3, 4, 5, 6]
    assert tiles.tolist() == [[0, 16, 20, 0], [16, 5, 36, 0], [43, 16, 0, 3], [59, 16, 16, 3], [75, 16, 32, 3], [91, 16, 48, 3]]
    assert b.rows_of((1, 2)).tolist() == list(range(21, 43))


@pytest.mark.parametrize("experts,top", [(5, 2), (4, 4), (1, 1), (7, 1)])
def test_router_bias_and_weights_over_the_chosen(experts, top):
    g = torch.Generator().manual_seed(experts)
    z, b = torch.randn(30, experts, generator=g), torch.randn(experts, generator=g)
    probs, idx = grouped.route_topk(z, top, renorm=True, shift=b)
    best, which = torch.topk(z + b, top, dim=-1)
    assert torch.equal(idx, which)
    torch.testing.assert_close(probs, torch.softmax(best, -1))


def test_experts_join_what_runs_beside_them():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    rows, dest, wts, base, res, w = r(9, 12), torch.tensor([3, 8, -1, 0, 5, 5], dtype=torch.int32), r(3, 2), r(3, 12), r(3, 12), r(12)
    want = res + base + torch.stack([wts[0, 0] * rows[3] + wts[0, 1] * rows[8], wts[1, 1] * rows[0], wts[2].sum() * rows[5]])
    h, out = stream.stream_norm(stream.ExpertSum(rows, dest, wts, base=base), res, w, 0.1, kind="layer", gain=0.3)
    torch.testing.assert_close(out, want)
    torch.testing.assert_close(h, 0.3 * O.layer_norm(want, w, 0.1))


def test_fused_matrices_hold_every_tensor_once():
    for model in O.MODELS.values():
        tensors = O.random_tensors(model)
        for i, spec in enumerate(ModelConfig.from_hf(model[0], O.shapes(tensors)).layer_specs):
            lay = LayerProjections(spec)
            mine = {k[len(f"l{i}.") :]: v for k, v in O.shapes(tensors).items() if k.startswith(f"l{i}.") and not k.endswith("norm1")}
            want = {k: v for k, v in mine.items() if not k.startswith(("mlp.e", "mlp.router"))}
            assert lay.tensors(model[0]["width"]) == want
            for ranges, total in ((lay.ins, lay.in_rows), (lay.outs, lay.out_cols)):
                used = sorted(ranges.values())
                assert all(a + n <= b for (a, n), (b, _) in zip(used, used[1:] + [(total, 0)]))


# ------------------------------------------------------------------------------------ whole models
def test_prompt_portions_and_decoding_agree_with_the_definition(case):
    model, tensors, tokens, want = case
    layers = []
    O.forward(model[0], tensors, tokens[:20], torch.float64, layers)
    for ps in (4, 16):
        e = make_engine(model, tensors, page_size=ps)
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
            assert len(e.kv.allocator.free) == free and len(e.free_slots) == 4
        assert e.stats["decode_steps"] > 70  # single tokens take the decode step


def test_unequal_batches_equal_each_request_alone(case):
    """Portions beside single tokens, streams that pause, streams that end and whose pages and slots the next ones take."""
    model, tensors, _, _ = case
    config = model[0]
    e = make_engine(model, tensors, num_pages=1 + 4 * 4, page_size=16)  # room for four streams of 64 tokens, no more
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
    model, tensors, _, _ = case
    config = model[0]
    prompts = [O.random_tokens(config, n, seed=20 + n) for n in (37, 1, 18, 50, 5)]
    steps = [12, 30, 9, 4, 40]
    e = make_engine(model, tensors, chunked_prefill_size=13, max_prefill_tokens=21, max_running_requests=3)
    reqs = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
    for p, n, r in zip(prompts, steps, reqs):
        assert len(r.output_ids) == n
        picks = O.forward(config, tensors, p + r.output_ids).log_softmax(-1)[len(p) - 1 : -1]
        assert torch.equal(picks.argmax(-1), torch.tensor(r.output_ids))
        want = picks.gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
        assert float((want - torch.tensor(r.output_logprobs)).abs().max()) < 1e-3
    again = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
    assert [r.output_ids for r in again] == [r.output_ids for r in reqs]
    assert again[0].num_cached_tokens == 32 and again[3].num_cached_tokens == 48  # whole pages come from the prefix cache
    r = e.generate([prompts[0]], [dict(max_new_tokens=0)], logprob_start_len=0)[0]  # prompt log-probs
    lp = O.forward(config, tensors, prompts[0]).log_softmax(-1)[:-1].gather(1, torch.tensor(prompts[0][1:])[:, None])[:, 0]
    assert float((lp - torch.tensor(r.input_logprobs[1:])).abs().max()) < 1e-3


def test_generation_under_page_pressure(case):
    model, tensors, _, _ = case
    prompts = [O.random_tokens(model[0], 30, seed=40 + i) for i in range(3)]
    sp = [dict(max_new_tokens=40, temperature=0, ignore_eos=True)] * 3
    roomy = make_engine(model, tensors, num_pages=64, page_size=8).generate(prompts, sp)
    tight = make_engine(model, tensors, num_pages=1 + 16, page_size=8)  # 128 tokens for 3 x 70: requests are retracted
    assert [r.output_ids for r in tight.generate(prompts, sp)] == [r.output_ids for r in roomy]


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding(name):
    model = O.MODELS[name]
    tensors, tokens = O.random_tensors(model, seed=2), O.random_tokens(model[0], 220, seed=3)
    want = O.forward(model[0], tensors, tokens)
    assert O.error(feed_all(make_engine(model, tensors), [9], tokens), want) < TOL


def _marked(mixer, rows=None):
    """One layer in which token 38 is a key that the query of token 39 matches and nothing else does."""
    model = O.model(48, 40, [(dict(mixer, **({"_rows": rows} if rows else {})), None)])
    t = O.random_tensors(model, seed=3, sharp=1.0)
    # coordinate 0 of the stream marks token 38, coordinate 1 token 39
    t["embed"][:, :2] = 0.0
    t["embed"][38, 0] = t["embed"][39, 1] = 40.0
    t["embed.norm"][:], t["l0.norm1"][:] = 1.0, 1.0
    return model, t


def _mark_heads(t, q_col=12, H_dim=16):
    for mark, x in enumerate("kq"):
        w = t[f"l0.mix.{x}"].view(-1, H_dim, 48)
        w.mul_(0.05)
        w[:, :, :2] = 0.0
        w[:, q_col, mark] = 20.0
        t[f"l0.mix.{x}.norm"][:] = 1.0


@pytest.mark.parametrize("cut", [0, 60])
@pytest.mark.parametrize("back", [3, 97, 146])
def test_a_key_far_back_is_found(cut, back):
    """The answer must move with the value stored at the one matching key, whether the prompt is one portion or the query is a
    decoded token; with a learned bias, far keys count by the last row of the table."""
    biased = _marked(O.biased(4, 2, 16, 16, 8, 30, scale=4.0, cap=30.0))
    _mark_heads(biased[1])
    lat = _marked(O.latent(3, 16, 4, 16, 8, 24, O.yarn_rot(4, 100.0), scale=6.0))
    t = lat[1]
    t["l0.mix.dq"].mul_(0.05)
    t["l0.mix.dkv"].mul_(0.05)
    t["l0.mix.dq"][0, 1], t["l0.mix.dkv"][0, 0] = 20.0, 20.0  # the latents' first coordinates carry the marks
    t["l0.mix.uq"].view(3, 20, 8)[:, 5, 0] = 6.0
    t["l0.mix.uk"].view(3, 16, 24)[:, 5, 0] = 6.0
    for model, tensors in (biased, lat):
        n = 150
        tokens = [x % 38 for x in O.random_tokens(model[0], n, seed=1)]
        tokens[n - 1 - back], tokens[-1] = 38, 39
        want = O.forward(model[0], tensors, tokens)
        other = list(tokens)
        other[n - 1 - back] = 5
        assert O.error(O.forward(model[0], tensors, other)[-1:], want[-1:]) > 0.1  # the far key decides
        for ps in (4, 64):
            e = make_engine(model, tensors, page_size=ps, num_pages=256 // ps + 1)
            assert O.error(feed_all(e, [n - cut], tokens), want) < TOL


@pytest.mark.parametrize("size", [5, 16, 33])
def test_edges_of_chunks(size):
    """A matching key just inside the query's chunk decides, one just outside must not, in prompts and in decoding."""
    model, tensors = _marked(O.chunked(4, 2, 16, size, O.yarn_rot(8, 100.0), scale=4.0, cap=30.0))
    _mark_heads(tensors)
    tensors["l0.mix.q.b"].zero_()
    tensors["l0.mix.k.b"].zero_()
    edge = 4 * size
    for q in (edge, edge + size - 1):
        for key, inside in ((edge, True), (edge - 1, False)):
            if key == q:
                continue
            tokens = [x % 38 for x in O.random_tokens(model[0], q + 1, seed=1)]
            tokens[key], tokens[q] = 38, 39
            want, other = O.forward(model[0], tensors, tokens), list(tokens)
            other[key] = 5
            moved = O.error(O.forward(model[0], tensors, other)[-1:], want[-1:])
            assert moved > 0.1 if inside else moved < 1e-12
            for ps in (4, 16):
                for cuts in ([q + 1], [q], [q - 1, 2], [edge - 1, 2]):
                    e = make_engine(model, tensors, page_size=ps, num_pages=512 // ps + 1)
                    assert O.error(feed_all(e, cuts, tokens), want) < TOL


def _patch(name, fn):
    return lambda mp, c, t: mp.setattr(O, name, fn(getattr(O, name)))


def _edit(layer, **kw):
    return lambda mp, c, t: c["layers"][layer]["mixer"].update(kw)


def _tensor(name, fn):
    return lambda mp, c, t: t.update({name: fn(t[name])})


MISTAKES = {  # of the model "odd": biased, latent, chunked
    "eps": lambda mp, c, t: c["norm"].update(eps=c["norm"]["eps"] * 3),
    "norm keeps the mean": _patch("layer_norm", lambda f: lambda x, w, eps: x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w),
    "logit factor": lambda mp, c, t: c.update(logit_scale=c["logit_scale"] * 1.01),
    "embedding not normed": _tensor("embed.norm", lambda x: torch.ones_like(x)),
    "no cap": _patch("soft_cap", lambda f: lambda s, cap: s),
    "cap": _edit(0, softcap=10.0),
    "bias before the cap": _patch("attend", lambda f: lambda q, k, v, scale, see, cap=None, bias=None: _bias_inside(q, k, v, scale, see, cap, bias)),
    "bias scaled": _tensor("l0.mix.rel", lambda x: x * 10**-0.5),
    "far distance": _edit(0, bias_max=11),
    "buckets one early": _patch("bucket", lambda f: lambda n, rows, far: f(n + 1, rows, far)),
    "buckets one late": _patch("bucket", lambda f: lambda n, rows, far: f(max(n - 1, 0), rows, far)),
    "chunk": _edit(2, mask=dict(size=8)),
    "a window for a chunk": _patch("chunk_mask", lambda f: lambda T, s: O.causal(T) & ~torch.ones(T, T, dtype=torch.bool).tril(-s)),
    "chunks counted from the portion": _patch("chunk_mask", lambda f: lambda T, s: f(T + 31, s)[31:, 31:]),
    "scale": _edit(1, scale=0.27),
    "norm per head": _patch("rms", lambda f: lambda x, w, eps: torch.cat([f(a, b, eps) for a, b in zip(x.split(10, -1), w.split(10, -1))], -1) if x.shape[-1] in (30, 60) else f(x, w, eps)),
    "values are the normed keys": _tensor("l2.mix.k.b", lambda x: x * 1.05),
    "no query bias": _tensor("l2.mix.q.b", torch.zeros_like),
    "pairs next to each other": _patch("rotate_halves", lambda f: lambda x, r: f(x[..., [0, 2, 4, 1, 3, 5] + list(range(6, x.shape[-1]))], r)[..., [0, 3, 1, 4, 2, 5] + list(range(6, x.shape[-1]))]),
    "no stretching": _patch("yarn", lambda f: lambda d, b, s: (f(d, b, None)[0], f(d, b, s)[1])),
    "no factor of the cosines": _patch("yarn", lambda f: lambda d, b, s: (f(d, b, s)[0], 1.0)),
    "a position late after 40 tokens": _patch("rotate_halves", lambda f: lambda x, r: torch.cat([f(x, r)[:40], f(torch.cat([x[:1], x]), r)[41:]])),
    "shared key normed": _patch("latent_attention", lambda f: lambda h, W, m, eps: f(h, lambda n: W(n) * (1.0 if n != "dkv" else _last(W(n), m["rot_dim"])), m, eps)),
    "latent not normed": _tensor("l1.mix.dkv.norm", lambda x: x * 1.03),
    "query latent norm": _tensor("l1.mix.dq.norm", torch.ones_like),
    "gate per channel": _tensor("l1.mix.g", lambda x: x.roll(1, 0)),
    "gate per head": _tensor("l2.mix.g", lambda x: x.roll(1, 0)),
    "router bias after the choice": _tensor("l0.mlp.router.b", torch.zeros_like),
    "weights over all experts": _patch("experts", lambda f: lambda h, W, m: _all_softmax(h, W, m)),
    "no shared expert": _tensor("l1.mlp.shared.down", torch.zeros_like),
    "sequential layer": _patch("experts", lambda f: lambda h, W, m: f(h * 1.02, W, m)),
    "value heads": _tensor("l0.mix.v", lambda x: x.roll(14, 0)),
}  # fmt: skip


def _bias_inside(q, k, v, scale, see, cap, bias):
    out = []
    for h in range(q.shape[1]):
        g = h // (q.shape[1] // k.shape[1])
        s = (q[:, h] @ k[:, g].t()) * scale + (0 if bias is None else bias[h])
        s = s if cap is None else cap * torch.tanh(s / cap)
        out.append(torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g])
    return torch.stack(out, 1)


def _last(w, n):
    f = torch.ones(w.shape[0], 1, dtype=w.dtype)
    f[-n:] = 0.8
    return f


def _all_softmax(h, W, f):
    z = h @ W("router").t() + W("router.b")
    weight, which = torch.topk(torch.softmax(z, -1), f["router"]["top"], dim=-1)
    ff = lambda e, x: O.feed_forward(x, W(e + ".gate"), W(e + ".up"), W(e + ".down"))  # noqa: E731
    y = torch.stack([sum(weight[t, j] * ff(f"e{int(which[t, j])}", h[t]) for j in range(weight.shape[1])) for t in range(len(h))])
    return y + ff("shared", h)


@pytest.fixture(scope="module")
def odd():
    model = O.MODELS["odd"]
    tensors, tokens = O.random_tensors(model, seed=1), O.random_tokens(model[0], 60, seed=1)
    got = feed_all(make_engine(model, tensors), [31, 2], tokens)
    assert O.error(got, O.forward(model[0], tensors, tokens)) < TOL
    return tensors, tokens, got


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_in_the_definition_shows(mistake, odd, monkeypatch):
    """The comparison is sharp: with one thing wrong in the definition the engine no longer agrees with it."""
    tensors, tokens, got = odd
    config, tensors = copy.deepcopy(O.MODELS["odd"][0]), dict(tensors)
    MISTAKES[mistake](monkeypatch, config, tensors)
    monkeypatch.setattr(O, "MIXERS", {k: getattr(O, v.__name__, v) for k, v in O.MIXERS.items()})  # patched functions are found by name
    if mistake == "shared key normed":
        monkeypatch.setitem(O.MIXERS, "latent_attention", O.latent_attention)
    assert O.error(got, O.forward(config, tensors, tokens)) > 5 * TOL


# ------------------------------------------------------------------------------------ configuration, loading, cache
def test_configuration_round_trip():
    for model in O.MODELS.values():
        tensors = O.random_tensors(model)
        cfg = ModelConfig.from_hf(model[0], O.shapes(tensors))
        assert cfg.num_params() == sum(v.numel() for v in tensors.values())
        written = json.loads(json.dumps(cfg.to_hf_dict()))
        assert ModelConfig.from_hf(written) == cfg  # carries the distance buckets
        for layer in written["layers"]:
            layer["mixer"].pop("bias_rows", None)
        assert written == model[0]
        assert [LayerSpec.of(s.to_dict()) for s in cfg.layer_specs] == cfg.layer_specs
    with pytest.raises(ValueError, match="rows"):
        ModelConfig.from_hf(O.MODELS["single"][0])
    bad = copy.deepcopy(O.MODELS["single"][0])
    bad["layers"][1]["type"] = "delta"
    with pytest.raises(ValueError, match="mixer"):
        ModelConfig.from_hf(bad, O.shapes(O.random_tensors("single")))
    bad = copy.deepcopy(O.MODELS["single"][0])
    bad["layers"][0]["mlp"]["kind"] = "dense"
    with pytest.raises(ValueError, match="feed-forward"):
        ModelConfig.from_hf(bad, O.shapes(O.random_tensors("single")))
    with pytest.raises(ValueError, match="layer_specs"):
        ModelConfig(num_layers=1, hidden_size=8, num_attention_heads=1, num_query_groups=1, ffn_hidden_size=8, vocab_size=8, logit_scale=2.0)


def test_mechanism_parameters_that_do_not_fit_are_refused():
    for kw in (dict(chunk=0), dict(softcap=-1.0), dict(distance_bias="linear"), dict(distance_bias="geometric", softcap=5.0), dict(norm_over="all"),
               dict(gate="token"), dict(tied_values=True)):  # fmt: skip
        with pytest.raises(ValueError):
            AttentionSpec(4, 2, 8, 16, 1.0, **kw)
    with pytest.raises(ValueError, match="rotated part"):
        LatentSpec(2, 8, 4, 8, 6, 12, 1.0, RotarySpec(6, 1e4))
    with pytest.raises(ValueError, match="gate"):
        LatentSpec(2, 8, 4, 8, 6, 12, 1.0, RotarySpec(4, 1e4), "head")
    with pytest.raises(ValueError, match="gate"):
        LayerSpec(AttentionSpec(1, 1, 8, 8, 1.0), FeedForwardSpec(8, "silu", experts=2, shared_ff=8, shared_gate=True), parallel_ff=True)


def test_loader_refuses_what_the_model_does_not_have():
    model = O.MODELS["mixed"]
    e = make_engine(model, O.random_tensors(model))
    z = torch.zeros(96, 96)
    for name in ("l0.norm2", "l1.mlp.up", "l0.mix.q", "l1.mix.v", "l2.mix.g", "l0.mix.q.b", "l2.mix.k.b", "l0.mlp.e9.up", "l2.mlp.shared.up", "head", "l9.norm1", "x"):
        assert e.update_weights([(name, z)]) == [name]
    with pytest.raises(ValueError, match="shape"):
        e.update_weights([("l0.mix.o", z)])
    assert set(e.weights.specified_tensors()) == set(O.random_tensors(model))


def test_weights_can_be_replaced():
    """A second load (a trainer's update) reaches everything that is derived from a tensor, the distance table included."""
    model = O.MODELS["mixed"]
    tokens = O.random_tokens(model[0], 40, seed=1)
    e = make_engine(model, O.random_tensors(model, seed=1))
    feed_all(e, [30], tokens)
    second = O.random_tensors(model, seed=2)
    e.update_weights(second.items())
    assert O.error(feed_all(e, [30], tokens), O.forward(model[0], second, tokens)) < TOL


def test_presets():
    for name in ("zetizen-a3b", "zetizen-tiny"):
        cfg = get_preset(name)
        assert cfg.model_arch == "Zetizen" and {type(s.mixer).__name__ for s in cfg.layer_specs} == {"AttentionSpec", "LatentSpec"}
        assert ModelConfig.from_hf(cfg.to_hf_dict()) == cfg
    e = Engine(get_preset("zetizen-tiny"), ServerArgs(page_size=16, max_running_requests=2, context_length=128), device="cpu", num_pages=20)
    e.weights.init_random(0)
    assert len(e.generate([[1, 2, 3]], [dict(max_new_tokens=5, temperature=0, ignore_eos=True)])[0].output_ids) == 5


def test_the_parts_serve_other_designs():
    """A sequential layer with chunked, capped, biased attention that has neither norms nor gates, one with a gate per channel and a
    window, a latent mixer without a gate, a mixture behind a mixer with a router bias and an untied head."""
    from slime_b200.models.layer_spec import flat_sizes

    dist = DistanceBiasSpec(8, 20)
    specs = [LayerSpec(AttentionSpec(4, 2, 8, 12, 0.5, chunk=9, softcap=3.0, distance_bias=dist), FeedForwardSpec(20, "silu")),
             LayerSpec(AttentionSpec(2, 1, 8, 8, 0.4, window=7, keep_first=2, gate="channel"), FeedForwardSpec(12, "relu2", False, 4, 2, renorm=True, router_bias=True)),
             LayerSpec(LatentSpec(2, 8, 4, 6, 10, 12, 0.4, RotarySpec(4, 50.0)))]  # fmt: skip
    cfg = ModelConfig(**dict(flat_sizes(specs), layer_specs=specs, hidden_size=16, vocab_size=30, model_arch="Other", tie_word_embeddings=False))
    e = Engine(cfg, ServerArgs(page_size=8, max_running_requests=2, context_length=64), device="cpu", num_pages=17)
    names = e.weights.specified_tensors()
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(*s, generator=g) * 0.5 for n, s in names.items()}
    assert not e.update_weights(t.items()) and "head" in t and "l1.mlp.router.b" in t
    tokens = O.random_tokens(dict(vocab=30), 40)
    rms = lambda x, n: O.rms(x, t[n], 1e-6)  # noqa: E731
    x, T = t["embed"][tokens], len(tokens)
    heads = lambda h, i, *c: [(h @ t[f"l{i}.mix.{n}"].t()).view(T, c[j], -1) for j, n in enumerate("qkv")]  # noqa: E731
    h = rms(x, "l0.norm1")
    x = x + O.attend(*heads(h, 0, 4, 2, 2), 0.5, O.chunk_mask(T, 9), 3.0, O.distance_bias(t["l0.mix.rel"], T, 20)).flatten(1) @ t["l0.mix.o"].t()
    x = x + O.feed_forward(rms(x, "l0.norm2"), t["l0.mlp.gate"], t["l0.mlp.up"], t["l0.mlp.down"])
    h = rms(x, "l1.norm1")
    see = O.causal(T) & (~torch.ones(T, T, dtype=torch.bool).tril(-7) | (torch.arange(T) < 2)[None, :])
    y = O.attend(*heads(h, 1, 2, 1, 1), 0.4, see).flatten(1) * torch.sigmoid(h @ t["l1.mix.g"].t())
    x = x + y @ t["l1.mix.o"].t()
    h = rms(x, "l1.norm2")
    top, which = torch.topk(h @ t["l1.mlp.router"].t() + t["l1.mlp.router.b"], 2, dim=-1)
    one = lambda e, v: torch.relu(v @ t[f"l1.mlp.e{e}.up"].t()) ** 2 @ t[f"l1.mlp.e{e}.down"].t()  # noqa: E731
    x = x + torch.stack([sum(w * one(int(e), v) for w, e in zip(ws, es)) for v, ws, es in zip(h, torch.softmax(top, -1), which)])
    h = rms(x, "l2.norm1")
    W = lambda n: torch.zeros(12, 16) if n == "g" else t["l2.mix." + n]  # noqa: E731
    m = dict(heads=2, dim=8, rot_dim=4, kv_rank=12, scale=0.4, rot=dict(dims=4, base=50.0))
    turn = O.rotate_halves
    pairs = lambda v, r: turn(v[..., [0, 2, 1, 3]], r)[..., [0, 2, 1, 3]]  # noqa: E731
    O.rotate_halves = pairs
    try:
        x = x + 2 * O.latent_attention(h, W, m, 1e-6)  # sigmoid(0) halves
    finally:
        O.rotate_halves = turn
    want = rms(x, "final.norm") @ t["head"].t()
    assert O.error(feed_all(e, [11, 2], tokens), want) < TOL


def test_trainer_says_that_it_cannot_train_this():
    from slime_b200.models.gpt import GPTModel

    model = O.MODELS["single"]
    with pytest.raises(NotImplementedError, match="rollout engine only"):
        GPTModel(ModelConfig.from_hf(model[0], O.shapes(O.random_tensors(model))), dtype=torch.float32, device="cpu")


@pytest.mark.parametrize("name", ["mixed", "even"])
def test_hand_over_and_host_tier(name):
    """Keys, values and latents travel between engines, and evicted pages come back from host memory."""
    model = O.MODELS[name]
    tensors, prompt = O.random_tensors(model, seed=8), O.random_tokens(model[0], 45, seed=8)
    sp = dict(max_new_tokens=10, temperature=0, ignore_eos=True)
    a, b = make_engine(model, tensors), make_engine(model, tensors)
    want = a.generate([prompt], [sp])[0]
    pre = a.generate([prompt], [sp], prefill_only=True)[0]
    r = b.import_request(prompt, pre.output_ids[0], pre.output_logprobs[0], pre.kv_export, sp)
    while not r.finished():
        b.step()
    assert r.output_ids == want.output_ids
    small = make_engine(model, tensors, num_pages=9, enable_hierarchical_cache=True, hicache_ratio=4.0)
    small.generate([prompt], [sp])
    for i in range(3):
        small.generate([O.random_tokens(model[0], 60, seed=60 + i)], [sp])
    again = small.generate([prompt], [sp])[0]
    assert again.output_ids == want.output_ids and small.kv.allocator.host_tier.hits > 0


def test_replay_writes_the_wanted_logits(tmp_path):
    from safetensors.torch import save_file

    from slime_b200.engine import trace

    model = O.MODELS["mixed"]
    config, tensors = model[0], O.random_tensors(model, seed=4)
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
    for gone in ("l0.mix.uk", "l1.mix.q.b", "l2.mlp.router.b", "embed.norm"):
        save_file({k: v for k, v in tensors.items() if k != gone}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ValueError, match="missing"):
            trace.load_engine(str(tmp_path), "float32", 128, 64, 4, torch.device("cpu"))


def _rank_main(rank, port, model, tensors, tokens, want, ep):
    import torch.distributed as dist

    torch.set_num_threads(1)
    dist.init_process_group("gloo", init_method=f"tcp://127.0.0.1:{port}", rank=rank, world_size=2)
    e = Engine(ModelConfig.from_hf(model[0], O.shapes(tensors)), ServerArgs(page_size=16, max_running_requests=4, context_length=128, ep_size=ep),
               device="cpu", num_pages=16, tp_group=dist.group.WORLD, tp_size=2, tp_rank=rank)  # fmt: skip
    assert not e.update_weights(tensors.items())
    assert O.error(feed_all(e, [17, 2, 20], tokens), want) < TOL
    dist.destroy_process_group()


@pytest.mark.parametrize("ep", [1, 2])
def test_two_tensor_parallel_ranks(ep):
    import socket

    model = O.model(48, 70, [(O.biased(4, 2, 16, 24, 8, 20), O.moe(6, 3, 24, 20)), (O.chunked(4, 2, 12, 11, O.yarn_rot(8)), O.moe(4, 1, 16)),
                             (O.latent(6, 8, 4, 16, 12, 20), O.moe(2, 2, 8, 10))])  # fmt: skip
    tensors, tokens = O.random_tensors(model, seed=3), O.random_tokens(model[0], 44, seed=3)
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    want = O.forward(model[0], tensors, tokens)
    torch.multiprocessing.spawn(_rank_main, args=(port, model, tensors, tokens, want, ep), nprocs=2)
    with pytest.raises(ValueError, match="divide"):
        t = O.random_tensors("odd")
        Engine(ModelConfig.from_hf(O.MODELS["odd"][0], O.shapes(t)), ServerArgs(), device="cpu", num_pages=4, tp_size=2)

"""Zetizen's kernels and models on a GPU, bf16 and full precision, against the plain definition (``zetizen_oracle``)."""

import json
import os
import subprocess
import sys

import pytest
import torch
import zetizen_oracle as O

from slime_b200.engine.engine import Engine
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig
from slime_b200.models.layer_spec import DistanceBiasSpec, RotarySpec, YarnSpec
from slime_b200.ops import grouped, latent, stream
from slime_b200.ops import window_attention as wa

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 2e-4, "bfloat16": 5e-2}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=["bfloat16", "float32"])
def dtype(request):
    return request.param


def _close(got, want, dtype, what=""):
    """Relative to the result's size: bf16 rounds the output and the operands of the second product."""
    err = (got.double().cpu() - want.double()).abs().max() / want.double().abs().max()
    assert float(err) < {"float32": 3e-5, "bfloat16": 1.5e-2}[dtype], (what, float(err))


def _rand(g, *shape, dtype, gain=1.0):
    """Values that bf16 holds, in either precision."""
    return (torch.randn(*shape, generator=g) * gain).bfloat16().to(getattr(torch, dtype))


# ------------------------------------------------------------------------------------------------ kernels
@pytest.mark.parametrize("H,G,D,DV,dims,tied", [(8, 2, 64, 64, 32, True), (6, 3, 24, 40, 0, False), (32, 8, 128, 128, 128, True), (3, 3, 10, 14, 6, False),
                                                (1, 1, 16, 16, 4, True)])  # fmt: skip
def test_heads_normed_over_the_projection(kernels, H, G, D, DV, dims, tied, dtype):
    g, T = torch.Generator().manual_seed(D), 37
    x = _rand(g, T, (H + G) * D + G * DV + 8, dtype=dtype)
    wq, wk = _rand(g, H * D, dtype=dtype), _rand(g, G * D, dtype=dtype)
    q, k = x[:, : H * D], x[:, H * D : (H + G) * D]
    v = k if tied else x[:, (H + G) * D : (H + G) * D + G * DV]
    rot = O.yarn_rot(dims, 500.0) if dims else None
    want_q, want_k = O.rms(q.double(), wq.double(), 1e-3).view(T, H, D), O.rms(k.double(), wk.double(), 1e-3).view(T, G, D)
    if dims:
        want_q, want_k = O.rotate_halves(want_q, rot), O.rotate_halves(want_k, rot)
    spec = RotarySpec(dims, 500.0, False, YarnSpec(**rot["scaling"])) if dims else None
    table = stream.rotary_table(T, dims, 500.0, DEV, frequencies=spec.frequencies(), gain=spec.gain()) if dims else None
    kc, vc = (torch.zeros(64, G, w, dtype=x.dtype, device=DEV) for w in (D, D if tied else DV))
    slots = torch.randperm(64, generator=g)[:T].int()
    slots[5] = -1  # a row without a place
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    xd = x.to(DEV)
    cut = lambda t, like: t[:, like.storage_offset() : like.storage_offset() + like.shape[1]]  # noqa: E731
    got = stream.place_heads(cut(xd, q), cut(xd, k), cut(xd, v), slots.to(DEV), kc, vc, q_norm=wq.to(DEV), k_norm=wk.to(DEV), eps=1e-3, table=table,
                             positions=pos, interleaved=False)  # fmt: skip
    rows = [t for t in range(T) if t != 5]
    _close(got, want_q, dtype)
    _close(kc.cpu()[slots[rows].long()], want_k[rows], dtype)
    assert torch.equal(vc.cpu()[slots[rows].long()].flatten(1), v[rows])
    assert float(kc.float().abs().sum(dim=(1, 2)).count_nonzero()) == T - 1
    if not dims and H > 1:  # parts of a projection: the sums come from outside
        half = H // 2 * D
        sums = stream.head_sums(x[:, : H * D].to(DEV), k.to(DEV))
        xd = x.to(DEV)
        part = stream.place_heads(xd[:, :half], cut(xd, k), cut(xd, v), slots.to(DEV), kc, vc, q_norm=wq[:half].to(DEV), k_norm=wk.to(DEV), eps=1e-3,
                                  sums=(sums, (H * D, G * D)))  # fmt: skip
        _close(part, want_q[:, : H // 2], dtype)


def _paged(g, lengths, ps, *tensors):
    """Rows of every request in scattered pages: (block table, pages, caches); what no row fills is NaN."""
    count = [-(-n // ps) for n in lengths]
    order = (torch.randperm(sum(count) + 3, generator=g)).tolist()
    pages = [[order.pop() for _ in range(c)] for c in count]
    caches = []
    for per in tensors:
        c = torch.full(((sum(count) + 3) * ps, *per[0].shape[1:]), float("nan"), dtype=per[0].dtype)
        for p, rows in zip(pages, per):
            i = torch.arange(len(rows))
            c[torch.tensor(p)[i // ps] * ps + i % ps] = rows
        caches.append(c.to(DEV))
    return pages, caches


SHAPES = [(8, 2, 64, 64, 64), (32, 8, 128, 128, 64), (6, 3, 24, 40, 16), (16, 1, 128, 64, 128), (4, 4, 64, 128, 32), (3, 3, 10, 14, 16), (4, 2, 160, 32, 64)]


@pytest.mark.parametrize("H,G,D,DV,ps", SHAPES)
@pytest.mark.parametrize("kind", ["near_bias", "far_bias", "bias_only", "chunk", "small_chunk", "cap_only"])
def test_capped_biased_and_chunked_attention(kernels, H, G, D, DV, ps, kind, dtype):
    g = torch.Generator().manual_seed(H + D)
    starts, counts = [0, 300, 77, 129], [261, 45, 1, 130]
    lengths = [s + n for s, n in zip(starts, counts)]
    q = [_rand(g, n, H, D, dtype=dtype) for n in lengths]
    k, v = ([_rand(g, n, G, w, dtype=dtype) for n in lengths] for w in (D, DV))
    scale, form, bias = 1.5 * D**-0.5, {}, None
    for r, n in enumerate(lengths):  # one far key that a late query must find, beside the chunk's and the window's edges
        k[r][n // 7] = (q[r][-1].view(G, H // G, D).float().mean(1) * 2).to(k[r].dtype)
    if kind in ("near_bias", "far_bias", "bias_only"):
        spec = DistanceBiasSpec(*{"near_bias": (16, 60), "far_bias": (64, 1500), "bias_only": (6, 11)}[kind])
        table = _rand(g, spec.rows, H, dtype="float32", gain=2.0)
        bias = O.distance_bias(table.double(), max(lengths), spec.far)
        form["bias"] = table[spec.by_distance()].contiguous().to(DEV)
    if kind != "bias_only":
        form["softcap"] = 3.0 if kind != "chunk" else 20.0
    if "chunk" in kind:
        form["chunk"] = 100 if kind == "chunk" else 7
    see = [O.chunk_mask(n, form["chunk"]) if "chunk" in form else O.causal(n) for n in lengths]
    want = [O.attend(q[r].double(), k[r].double(), v[r].double(), scale, see[r], form.get("softcap"), None if bias is None else bias[:, :n, :n])
            for r, n in enumerate(lengths)]  # fmt: skip
    pages, (kc, vc) = _paged(g, lengths, ps, k, v)
    batch = wa.ExtendBatch.build(pages, starts, counts, ps, DEV)
    rows = lambda x: torch.cat([a[s : s + n] for a, s, n in zip(x, starts, counts)])  # noqa: E731
    for gates in (0, 1, DV):
        gate = _rand(g, sum(counts), H * gates + 8, dtype=dtype)[:, : H * gates] if gates else None
        factor = torch.sigmoid(gate.double()).view(-1, H, gates) if gates else 1.0
        got = wa.window_extend(rows(q).to(DEV), kc, vc, batch, scale, gate=None if gate is None else gate.to(DEV), **form)
        _close(got, rows(want) * factor, dtype, gates)
    last = torch.stack([x[-1] for x in q]).to(DEV)
    table = batch.block_table
    seq = torch.tensor(lengths, dtype=torch.int32, device=DEV)
    for most in (None, 4096):
        gate = _rand(g, len(q), H, dtype=dtype)
        got = wa.window_decode(last, kc, vc, table, seq, seq - 1, ps, scale, max_context=most, gate=gate.to(DEV), **form)
        _close(got, torch.stack([w[-1] for w in want]) * torch.sigmoid(gate.double())[..., None], dtype, most)


LATENTS = [(6, 64, 32, 48, 96, 64), (16, 128, 64, 128, 512, 64), (40, 32, 16, 64, 192, 16), (3, 24, 8, 40, 320, 32), (3, 10, 6, 14, 22, 16),
           (128, 128, 64, 128, 512, 64), (2, 160, 64, 32, 64, 128), (20, 64, 64, 64, 64, 64), (5, 16, 6, 8, 34, 16)]  # fmt: skip


@pytest.mark.parametrize("H,D,r,DV,R,ps", LATENTS)
def test_latent_attention(kernels, H, D, r, DV, R, ps, dtype):
    g = torch.Generator().manual_seed(R + H)
    many = H > 32
    starts, counts = ([0, 140, 33], [70, 90, 3]) if many else ([0, 300, 77, 129, 500], [261, 65, 1, 130, 13])
    lengths = [s + n for s, n in zip(starts, counts)]
    rot, scale, R1 = O.yarn_rot(r, 200.0), (D + r) ** -0.5, 24
    T = sum(counts)
    table = stream.rotary_table(max(lengths) + 1, r, 200.0, DEV, frequencies=RotarySpec(r, 200.0, False, YarnSpec(**rot["scaling"])).frequencies(),
                                gain=YarnSpec(**rot["scaling"]).gain())  # fmt: skip
    up_q, up_kv = _rand(g, H * (D + r), R1, dtype=dtype, gain=R1**-0.5), _rand(g, H * (D + DV), R, dtype=dtype, gain=R**-0.5)
    L = latent.Latent(H, D, DV, R, scale, up_q.to(DEV), up_kv.to(DEV), table)
    q, down = [_rand(g, n, H, D + r, dtype=dtype, gain=2.0) for n in lengths], [_rand(g, n, R + r, dtype=dtype) for n in lengths]
    want, cached = [], []
    for n, x, c in zip(lengths, q, down):
        c = torch.cat([c[:, :R], O.rotate_halves(c[:, None, R:].double(), rot)[:, 0].to(c.dtype)], 1)  # as the cache holds it
        cached.append(c[:, None])
        x, c = x.double(), c.double()
        k = torch.cat([(c[:, :R] @ up_kv[: H * D].double().t()).view(n, H, D), c[:, None, R:].expand(n, H, r)], -1)
        qq = torch.cat([x[..., :D], O.rotate_halves(x[..., D:], rot)], -1)
        want.append(O.attend(qq, k, (c[:, :R] @ up_kv[H * D :].double().t()).view(n, H, DV), scale, O.causal(n)))
    pages, (cache,) = _paged(g, lengths, ps, cached)
    rows = lambda x: torch.cat([a[s : s + n] for a, s, n in zip(x, starts, counts)])  # noqa: E731
    wide = _rand(g, T, H * DV + 16, dtype=dtype)
    gate = wide[:, 8 : 8 + H * DV].unflatten(1, (H, DV))
    for gated in (False, True):
        out = torch.zeros(T, H * DV + 8, dtype=wide.dtype, device=DEV)
        view = out[:, : H * DV].unflatten(1, (H, DV))
        gd = wide.to(DEV)[:, 8 : 8 + H * DV].unflatten(1, (H, DV)) if gated else None
        latent.latent_extend(L, rows(q).to(DEV), cache, wa.ExtendBatch.build(pages, starts, counts, ps, DEV), gd, view)
        factor = torch.sigmoid(gate.double()) if gated else 1.0
        _close(view, rows(want) * factor, dtype, "extend")
        assert float(out[:, H * DV :].abs().max()) == 0
    batch = wa.ExtendBatch.build(pages, starts, counts, ps, DEV)
    last = torch.stack([x[-1] for x in q]).to(DEV)
    pos = torch.tensor(lengths, dtype=torch.int32, device=DEV) - 1
    for most in (max(lengths), 8192):  # one range of keys, and several of which most are empty
        out = torch.zeros(len(q), H, DV, dtype=wide.dtype, device=DEV)
        latent.latent_decode(L, last, cache, batch.block_table, pos, ps, most, gate[: len(q)].contiguous().to(DEV), out)
        _close(out, torch.stack([w[-1] for w in want]) * torch.sigmoid(gate[: len(q)].double()), dtype, "decode")


def test_latent_projections_into_the_cache(kernels, dtype):
    for R1, R, r in ((96, 128, 32), (24, 48, 16), (11, 19, 6), (1536, 512, 64)):
        g, T, eps = torch.Generator().manual_seed(R), 33, 1e-3
        rot = O.yarn_rot(r, 300.0)
        spec = RotarySpec(r, 300.0, False, YarnSpec(**rot["scaling"]))
        x = _rand(g, T, R1 + R + r + 16, dtype=dtype)
        dq, dkv = x[:, 8 : 8 + R1], x[:, 8 + R1 : 8 + R1 + R + r]
        wq, wk = _rand(g, R1, dtype=dtype), _rand(g, R, dtype=dtype)
        table = stream.rotary_table(T, r, 300.0, DEV, frequencies=spec.frequencies(), gain=spec.gain())
        cache, slots = torch.zeros(64, 1, R + r, dtype=x.dtype, device=DEV), torch.randperm(64, generator=g)[:T].int()
        slots[7] = -1
        xd = x.to(DEV)
        got = latent.latent_place(xd[:, 8 : 8 + R1], xd[:, 8 + R1 : 8 + R1 + R + r], wq.to(DEV), wk.to(DEV), eps, table,
                                  torch.arange(T, dtype=torch.int32, device=DEV), slots.to(DEV), cache)  # fmt: skip
        _close(got, O.rms(dq.double(), wq.double(), eps), dtype)
        want = torch.cat([O.rms(dkv[:, :R].double(), wk.double(), eps), O.rotate_halves(dkv[:, None, R:].double(), rot)[:, 0]], 1)
        rows = [t for t in range(T) if t != 7]
        _close(cache.cpu()[slots[rows].long(), 0], want[rows], dtype)


def test_experts_beside_a_mixer(kernels, dtype):
    """Router with a bias, weights over the chosen logits; their sum, the mixer's output, residual, norm and factor in one launch."""
    g, T, D, E, k = torch.Generator().manual_seed(3), 50, 96, 7, 3
    z, b = torch.randn(T, E, generator=g), torch.randn(E, generator=g)
    probs, idx = grouped.route_topk(z.to(DEV), k, renorm=True, raw_index=True, shift=b.to(DEV))
    top, which = torch.topk((z + b).double(), k, dim=-1)
    assert torch.equal(idx.cpu().long(), which)
    torch.testing.assert_close(probs.cpu().double(), torch.softmax(top, -1), atol=1e-6, rtol=1e-5)
    lay = grouped.DeviceLayout(idx, E)
    rows = _rand(g, lay.rows_padded, D, dtype=dtype)
    base, res, w = torch.randn(T, D, generator=g), torch.randn(T, D, generator=g), _rand(g, D, dtype=dtype)
    picked = rows.double()[lay.slot_dest.cpu().long()].view(T, k, D)
    want = res.double() + (picked * torch.softmax(top, -1)[..., None]).sum(1) + base.double()
    out = res.to(DEV)
    h, _ = stream.stream_norm(stream.ExpertSum(rows.to(DEV), lay.slot_dest, probs, base=base.to(DEV)), out, w.to(DEV), 1e-4, kind="layer", gain=0.37)
    _close(out, want, "float32")
    _close(h, O.layer_norm(want, w.double(), 1e-4) * 0.37, dtype)


# ------------------------------------------------------------------------------------------------- models
MODELS = dict(O.MODELS, wide=O.model(384, 1000, [  # tensor-core shapes throughout, several key tiles
    (O.biased(8, 2, 64, 128, 32, 128, cap=15.0), O.moe(16, 4, 128, 256)), (O.chunked(8, 4, 128, 100, O.yarn_rot(64, 5e5)), O.moe(8, 2, 64, 64)),
    (O.latent(4, 128, 64, 128, 192, 512), O.moe(8, 3, 64)), (O.latent(18, 64, 32, 64, 64, 160), None)], logit_scale=0.5))  # fmt: skip


def make_engine(model, tensors, dtype, num_pages=64, page_size=16, **kw):
    kw = {"max_running_requests": 4, "context_length": 512, "dtype": dtype, **kw}
    e = Engine(ModelConfig.from_hf(model[0], O.shapes(tensors)), ServerArgs(page_size=page_size, **kw), device="cuda", num_pages=num_pages)
    assert e.dtype == getattr(torch, dtype) and not e.update_weights(tensors.items())
    return e


def weights(model, seed, dtype):
    """bf16 values in either precision; gentler attention where bf16 rounding of q and k would swamp a sharp softmax, and routers
    that mostly follow their bias, so that rounding does not turn a close call between two experts."""
    t = O.random_tensors(model, seed=seed, sharp=2.5 if dtype == "float32" else 1.0)
    if dtype == "bfloat16":
        t.update({k: v * 0.02 for k, v in t.items() if k.endswith("mlp.router")})
        t.update({k: torch.arange(v.numel()).roll(v.numel() // 2) * 0.4 for k, v in t.items() if k.endswith("router.b")})
    return {k: v.bfloat16() for k, v in t.items()}


@pytest.mark.parametrize("name", sorted(MODELS))
def test_portions_and_decoding(kernels, name, dtype):
    model = MODELS[name]
    n = 300 if name == "wide" else 120
    tensors, tokens = weights(model, 5, dtype), O.random_tokens(model[0], n, seed=6)
    want = O.forward(model[0], tensors, tokens)
    for ps in (16, 64):
        e = make_engine(model, tensors, dtype, page_size=ps)
        for cuts in ([n], [n - 20], [2] * 30, [37, 3, 16, 2, 29], [64, 33]):
            req, at, out = e.open_stream("s"), 0, []
            for c in cuts + [1] * (n - sum(cuts)):
                out.append(e.feed([(req, tokens[at : at + c], list(range(c)))]))
                at += c
            e.close_stream(req)
            err = O.error(torch.cat(out).cpu(), want)
            assert err < TOL[dtype], (ps, cuts, err)
        assert e.runner.graphs  # single tokens were graph replays


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_mixed_batches_and_reused_pages(kernels, name, dtype):
    model = MODELS[name]
    config = model[0]
    tensors = weights(model, 7, dtype)
    e = make_engine(model, tensors, dtype, num_pages=1 + 4 * 8, page_size=16)  # four streams of 128 tokens
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
        err = O.error(torch.cat(got[i]), want[i])
        assert err < TOL[dtype], (i, err)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation(kernels, name, dtype):
    model = MODELS[name]
    config = model[0]
    tensors = weights(model, 9, dtype)
    e = make_engine(model, tensors, dtype, chunked_prefill_size=13, max_prefill_tokens=21, max_running_requests=3)
    prompts = [O.random_tokens(config, n, seed=20 + n) for n in (37, 1, 18, 50)]
    steps = [12, 30, 9, 25]
    for _ in range(2):  # the second time with graphs, and with prefixes from the cache
        reqs = e.generate(prompts, [dict(max_new_tokens=n, temperature=0, ignore_eos=True) for n in steps])
        for p, r in zip(prompts, reqs):
            lp = O.forward(config, tensors, p + r.output_ids).log_softmax(-1)[len(p) - 1 : -1]
            ids = torch.tensor(r.output_ids)[:, None]
            assert float((lp.gather(1, ids)[:, 0] - torch.tensor(r.output_logprobs)).abs().max()) < 8 * TOL[dtype]
            assert float((lp.max(-1).values - lp.gather(1, ids)[:, 0]).max()) < 8 * TOL[dtype]  # the best token, or a tie with it


def test_trace_run_program(kernels, tmp_path):
    from safetensors.torch import save_file

    model = O.MODELS["even"]
    config = model[0]
    tensors = weights(model, 4, "float32")
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

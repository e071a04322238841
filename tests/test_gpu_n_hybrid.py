"""Delta-net hybrids (Qwen3.5 layout) in the engine on a GPU, bf16, against the same engine in fp32 on the CPU."""

import pytest
import torch

from slime_b200.engine.engine import Engine
from slime_b200.engine.server_args import ServerArgs
from slime_b200.models.config import ModelConfig

pytestmark = pytest.mark.gpu


def _config(arch):
    return ModelConfig(num_layers=4, hidden_size=128, num_attention_heads=4, num_query_groups=2, kv_channels=64, ffn_hidden_size=192, vocab_size=300,
                       tie_word_embeddings=False, qk_layernorm=True, attention_output_gate=True, full_attention_interval=2, linear_num_key_heads=2,
                       linear_num_value_heads=4, linear_key_head_dim=32, linear_value_head_dim=48, model_arch=arch)  # fmt: skip


@pytest.mark.parametrize("arch", ["Qwen3_5ForCausalLM", "Qwen3NextForCausalLM"])
def test_portions_steps_and_generation(kernels, arch):
    make = lambda dev: Engine(_config(arch), ServerArgs(page_size=16, max_running_requests=3, context_length=256, chunked_prefill_size=32), device=dev, num_pages=64)  # noqa: E731,E501
    cpu, gpu = make("cpu"), make("cuda")
    cpu.weights.init_random(1, std=0.08)
    for a, b in zip(cpu.weights.tensors(), gpu.weights.tensors()):
        a.copy_(a.bfloat16())
        b.copy_(a)
    tokens = torch.randint(0, 300, (90,), generator=torch.Generator().manual_seed(2)).tolist()

    def feed(e, cuts):
        req, at, out = e.open_stream("s"), 0, []
        for n in cuts:
            out.append(e.feed([(req, tokens[at : at + n], list(range(n)))]).float().cpu())
            at += n
        e.close_stream(req)
        return torch.cat(out)

    want = feed(cpu, [90])
    for cuts in ([90], [60] + [1] * 30, [5, 2, 31, 1, 1, 50]):
        assert float((feed(cpu, cuts) - want).abs().max()) < 1e-3
        d = feed(gpu, cuts) - want
        err = d.pow(2).mean(-1).sqrt() / want.std()  # this family's residual stream is bf16: rounding shows in every row
        assert float(err.median()) < 3e-2 and float(err.max()) < 0.12, (cuts, float(err.median()), float(err.max()))
    prompts, sp = [tokens[:40], tokens[40:47], tokens[10:80], tokens[:3]], dict(max_new_tokens=20, temperature=0, ignore_eos=True)
    for p, r in zip(prompts, gpu.generate(prompts, [sp] * 4)):
        req = cpu.open_stream("g")
        lp = cpu.feed([(req, p + r.output_ids, list(range(len(p) - 1, len(p) + 19)))]).log_softmax(-1)
        cpu.close_stream(req)
        got = lp.gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
        assert float((got - torch.tensor(r.output_logprobs)).abs().max()) < 0.25 and float((lp.max(-1).values - got).max()) < 0.25
    assert len(gpu.states.free) == 3

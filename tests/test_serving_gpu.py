"""The serving engine on the device with the Llama family: ragged steps over the paged cache against the dense forward."""
import pytest
import torch

from ferrotorch_b200 import _native
from ferrotorch_b200.models.llama import LlamaConfig, LlamaForCausalLM
from ferrotorch_b200.models.serving import ContinuousBatcher, PagedStepper

pytestmark = pytest.mark.gpu


def _model(dtype, head_dim):
    torch.manual_seed(3)
    cfg = LlamaConfig(vocab_size=320, hidden_size=256, intermediate_size=384, num_hidden_layers=2, num_attention_heads=4,
                      num_key_value_heads=2, head_dim=head_dim, max_position_embeddings=512, initializer_range=0.08)
    return LlamaForCausalLM(cfg).to("cuda", dtype).eval()


@pytest.mark.parametrize("head_dim", [64, 128, 48])
@pytest.mark.parametrize("dtype,tol", [(torch.bfloat16, 0.04), (torch.float32, 1e-4)], ids=["bf16", "fp32"])
def test_ragged_steps_match_the_dense_forward(dtype, tol, head_dim):
    model = _model(dtype, head_dim)
    oracle = LlamaForCausalLM(model.config).to("cuda", torch.float32).eval()
    oracle.load_state_dict(model.state_dict())
    g = torch.Generator().manual_seed(1)
    toks = [torch.randint(0, 320, (n,), generator=g).tolist() for n in (300, 41, 150)]
    with torch.no_grad():
        want = [oracle(torch.tensor([t], device="cuda"))[0].double() for t in toks]
    for graph in (False, True):
        st = PagedStepper(model, 34, 16, 4, 512, cuda_graph=graph)
        slots, at = [st.admit() for _ in toks], [0, 0, 0]
        for sizes in ((129, 1, 2), (1, 30, 100), (128, 1, 1), (1, 1, 1), (41, 8, 46)):
            parts, rows = [], []
            for i, n in enumerate(sizes):
                parts.append((slots[i], toks[i][at[i]:at[i] + n], [n - 1]))
                at[i] += n
                rows.append(want[i][at[i] - 1])
            got, ref = st.feed(parts).double(), torch.stack(rows)
            assert float((got - ref).pow(2).mean(-1).sqrt().max() / ref.pow(2).mean().sqrt()) < tol
        assert at == [300, 41, 150] and _native.device_status(0) == 0
        assert (st.graph_replays > 0) == graph


def test_captured_decode_steps_give_the_tokens_of_eager_ones():
    model = _model(torch.bfloat16, 64)
    g = torch.Generator().manual_seed(2)
    prompts = [torch.randint(0, 320, (n,), generator=g).tolist() for n in (17, 3, 60, 9, 31)]
    eager = ContinuousBatcher(model, 64, 16, 4, 256, prefill_chunk=32).generate(prompts, 12)
    batcher = ContinuousBatcher(model, 64, 16, 4, 256, prefill_chunk=32, cuda_graph=True)
    assert batcher.generate(prompts, 12) == eager and batcher.stepper.graph_replays > 0

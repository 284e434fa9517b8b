"""The Bopudra decoder on its kernels, bf16 and fp32, against the plain oracle; the kernels alone at larger sizes."""
import pytest
import torch

import bopudra_cases as C
import bopudra_oracle as O
from planted_keys import check_planted_keys
from ferrotorch_b200 import _native
from ferrotorch_b200.nn.paged import PagedAttentionManager, PagedKVCache, RaggedBatch
from ferrotorch_b200.ops import functional as F
from ferrotorch_b200.ops import reference as R

pytestmark = pytest.mark.gpu
_DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
_cases: dict = {}


@pytest.fixture(params=[(n, d) for n in sorted(C.CASES) for d in _DTYPES], ids=lambda p: "%s-%s" % p)
def case(request):
    name, d = request.param
    if request.param not in _cases:
        _cases[request.param] = C.Case(name, _DTYPES[d], "cuda")
    yield _cases[request.param]
    assert _native.device_status(0) == 0


def test_whole_prompt(case):
    before = _native.launch_count()
    C.check_whole_prompt(case)
    assert _native.launch_count() - before >= 2 + 2 * len(case.cfg["layers"])


@pytest.mark.parametrize("block", [4, 8, 16, 64])
def test_portions_and_single_tokens(case, block):
    C.check_portions(case, block)


@pytest.mark.parametrize("graph", [False, True], ids=["eager", "graph"])
def test_unequal_requests_in_one_batch(case, graph):
    C.check_batches(case, cuda_graph=graph)


def test_long_prompts_and_long_decoding(case):
    toks = case.tokens(430, 71)
    want = O.forward(case.cfg, case.weights, toks)
    for cuts, kw in (([430], {}), ([3, 127, 2, 130, 1], {}), ([129, 1], dict(cuda_graph=True))):
        case.check(C.feed_all(case, cuts, toks, **kw), want, str(cuts))


def test_greedy_generation_through_the_scheduler(case):
    C.check_generation(case)
    b = C.check_generation(case, blocks=6, cuda_graph=True)
    assert b.stepper.graph_replays > 0 and b.stats.preemptions > 0


def test_residual_after_every_layer(case):
    toks = case.tokens(19, 9)
    _, want = O.forward(case.cfg, case.weights, toks, every_layer=True)
    st, seen = case.stepper(32), {}
    st.reserve(st.admit(), 19)
    case.model.paged_forward(RaggedBatch([(0, toks, 0, [])], "cuda"), st.cache, on_layer=lambda i, x: seen.update({i: x.clone()}))
    width = case.cfg["width"]
    for i, w in enumerate(want):
        got = seen[i].double().cpu()
        assert seen[i].dtype == torch.float32 and not got[:, width:].any()
        assert float((got[:, :width] - w).pow(2).mean().sqrt() / w.pow(2).mean().sqrt()) < case.tolerance


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("Hq,Hkv,D,Dv,block", [
    (6, 2, 16, 48, 8), (3, 3, 32, 16, 16), (5, 1, 48, 80, 4), (8, 2, 128, 128, 16), (8, 1, 64, 64, 32), (4, 4, 64, 64, 16),
    (12, 2, 112, 96, 64), (16, 1, 80, 128, 128), (14, 2, 128, 64, 256), (24, 1, 48, 32, 16), (40, 2, 64, 128, 8), (130, 1, 16, 16, 16),
    (4, 2, 160, 32, 16), (2, 1, 40, 24, 16), (6, 3, 32, 32, 12)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_attention_over_pages_sees_the_key_it_should(Hq, Hkv, D, Dv, block, dtype):
    if dtype == "fp32" and Hq * D > 1024:
        pytest.skip("the same kernel at a smaller size")
    check_planted_keys(Hq, Hkv, D, Dv, block, _DTYPES[dtype], "cuda", length=150 if Hq * D < 400 else 139)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("Hq,Hkv,D,Dv", [(8, 2, 128, 128), (6, 2, 96, 64), (4, 4, 64, 128)])
def test_prefill_kernel_long_portions(Hq, Hkv, D, Dv):
    # many tiles of several sequences at different contexts, scores that grow along the sequence (lazy rescale)
    torch.manual_seed(D + Dv)
    bs, plan = 16, [(700, 390), (1500, 257), (64, 64), (2, 2), (1030, 1029)]
    cache = PagedKVCache(1, Hkv, D, sum((n + bs - 1) // bs for n, _ in plan), len(plan), 1600, bs, v_head_dim=Dv)
    mgr = PagedAttentionManager(cache)
    entries, ks, vs = [], [], []
    for n, new in plan:
        s = mgr.add_sequence(n)
        k = (torch.randn(n, Hkv, D, device="cuda") * torch.linspace(0.3, 2.0, n, device="cuda").view(n, 1, 1)).bfloat16()
        v = torch.randn(n, Hkv, Dv, device="cuda").bfloat16()
        pages = torch.tensor(cache.pages_of(s), device="cuda")
        pad = len(pages) * bs - n
        cache.k[0][pages] = torch.nn.functional.pad(k, (0, 0, 0, 0, 0, pad)).view(-1, bs, Hkv, D)
        cache.v[0][pages] = torch.nn.functional.pad(v, (0, 0, 0, 0, 0, pad)).view(-1, bs, Hkv, Dv)
        entries.append((s, [0] * new, n - new, []))
        ks.append(k), vs.append(v)
    batch = RaggedBatch(entries, "cuda")
    q = torch.randn(batch.n_rows, Hq, D, device="cuda").bfloat16()
    out = cache.attend(0, q, batch)
    torch.cuda.synchronize()
    assert _native.device_status(0) == 0
    for (slot, row, start, n), k, v in zip(batch.spans, ks, vs):
        want, _ = R.attention(q[row:row + n][None], k[None], v[None], True, D ** -0.5, start)
        err = (out[row:row + n].float() - want[0].float()).abs().max().item()
        assert err < 4e-2, (slot, err)


@pytest.mark.parametrize("M", [1, 5, 64, 65, 128])
def test_small_batch_gemm_adds_to_the_residual_and_normalises(M):
    torch.manual_seed(M)
    N, K = 1032, 2056
    a, w = torch.randn(M, K, device="cuda").bfloat16(), (torch.randn(N, K, device="cuda") * K ** -0.5).bfloat16()
    x = torch.randn(M, N, device="cuda") * 3
    alpha, nw, nb = torch.tensor(0.6, device="cuda"), torch.randn(N, device="cuda"), torch.randn(N, device="cuda")
    want = x.double() + a.double() @ w.double().t()
    assert torch.allclose(F.linear_f32_out(a, w).double(), want - x.double(), atol=1e-4)
    h = F.residual_linear_(x, a, w, (alpha, nw, nb, 1.5))
    assert x.dtype == torch.float32 and torch.allclose(x.double(), want, atol=1e-4)
    wide = (torch.randn(20008, K, device="cuda") * K ** -0.5).bfloat16()       # fills the GPU without a split
    got = F.linear_f32_out(a, wide)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), a.double() @ wide.double().t(), atol=1e-4)
    assert torch.allclose(h.double(), (O.dynamic_tanh(want, 0.6, nw.double(), nb.double()) * 1.5), atol=3e-2, rtol=8e-3)


@pytest.mark.parametrize("rows,H", [(1, 8), (3, 2056), (700, 1032)])
def test_dynamic_tanh_kernel(rows, H):
    x, w, b = torch.randn(rows, H, device="cuda") * 2, torch.randn(H, device="cuda"), torch.randn(H, device="cuda")
    alpha = torch.tensor(-0.8, device="cuda")
    want = O.dynamic_tanh(x.double(), -0.8, w.double(), b.double())
    assert torch.allclose(F.dynamic_tanh(x, alpha, w, b).double(), want, atol=3e-6)
    ids = torch.randint(0, rows, (5,), device="cuda")
    got_x, h = F.embedding_dynamic_tanh(ids, x, alpha, w, b)
    assert torch.equal(got_x, x[ids]) and torch.allclose(h.double(), want[ids], atol=3e-6)
    xb = x.bfloat16()
    got_x, h = F.embedding_dynamic_tanh(ids, xb, alpha, w, b)
    assert torch.equal(got_x, xb[ids].float()) and h.dtype == torch.bfloat16


def test_query_temperature_far_into_a_sequence():
    # positions around exact multiples, as the kernel sees them
    pos = [0, 6, 7, 8, 8190, 8191, 8192, 57343, 57344, 99999, 1048575]
    for every in (1, 7, 8192):
        cache = PagedKVCache(1, 1, 16, 1, 1, 1 << 20, 1 << 20, dtype=torch.float32)
        cache.reserve(0, 1 << 20)
        batch = RaggedBatch([(0, [0], p, []) for p in pos], "cuda")
        packed = torch.ones(len(pos), 48, device="cuda")
        F.qkv_finish(packed, cache, 0, batch, q=(0, 16), k=(16, 16), v=(32, 16), temp_coef=0.7, temp_every=every)
        assert packed[:, 0].tolist() == pytest.approx([O.query_temperature(p, 0.7, every) for p in pos], rel=2e-6)


def test_model_with_wide_layers_matches_its_fp32_self():
    # sizes that take the CTA-pair and small-batch GEMMs, the fused norm of the split finalize pass and head size 128
    from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM
    from ferrotorch_b200.models.serving import PagedStepper

    cfg = BopudraConfig.uniform(2000, 1096, 3, 10, 2, 128, 1704, vdim=112)
    got = {}
    toks = torch.randint(0, 2000, (500,), generator=torch.Generator().manual_seed(5)).tolist()
    for dtype in (torch.float32, torch.bfloat16):
        model = BopudraForCausalLM(cfg, torch.float32, "cuda").random_(0.05)
        weights = {k: v.bfloat16().float() if "norm" not in k else v for k, v in model.checkpoint_tensors().items()}
        model = BopudraForCausalLM(cfg, dtype, "cuda")
        model.load_tensors(weights)
        st = PagedStepper(model, 40, 16, 4, 640, cuda_graph=dtype == torch.bfloat16)
        s = st.admit()
        rows = [st.feed([(s, toks[:410], [0, 127, 128, 409])])]
        rows += [st.feed([(s, toks[410 + 6 * i:416 + 6 * i], range(6))]) for i in range(5)]
        rows += [st.feed([(s, [t], [0])]) for t in toks[440:]]
        got[dtype] = torch.cat(rows).double()
    a, b = got[torch.float32], got[torch.bfloat16]
    err = (a - b).pow(2).mean(-1).sqrt() / a.pow(2).mean().sqrt()
    assert float(err.max()) < 0.03 and _native.device_status(0) == 0

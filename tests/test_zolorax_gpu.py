"""The Zolorax decoder on its kernels, bf16 and fp32, against the plain oracle; the kernels alone at larger sizes."""
import pytest
import torch

import decoder_cases as C
import zolorax_oracle as O
from zolorax_cases import CASES, Case
from ferrotorch_b200 import _native
from ferrotorch_b200.nn.packed_block import RotarySpec
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.ops import decoder as D
from ferrotorch_b200.ops import functional as F
from ferrotorch_b200.ops import reference as R
from planted_keys import check_planted_keys

pytestmark = pytest.mark.gpu
_DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
_cases: dict = {}


@pytest.fixture(params=[(n, d) for n in sorted(CASES) for d in _DTYPES], ids=lambda p: "%s-%s" % p)
def case(request):
    name, d = request.param
    if request.param not in _cases:
        _cases[request.param] = Case(name, _DTYPES[d], "cuda")
    yield _cases[request.param]
    assert _native.device_status(0) == 0


def _rnd(*shape, std=1.0, dtype=torch.float32):
    return (torch.randn(*shape, device="cuda") * std).to(dtype)


# ------------------------------------------------------------------ the model
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
    want = case.oracle(toks)
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


# ------------------------------------------------------------------ attention with window, sink and element gates
@pytest.mark.parametrize("Hq,Hkv,D,Dv,block,window", [
    (6, 2, 16, 48, 8, 20), (4, 4, 64, 64, 16, 33), (8, 2, 128, 128, 16, 64), (8, 1, 64, 64, 32, 1), (5, 1, 48, 80, 4, 50), (12, 2, 112, 96, 64, 128),
    (14, 2, 128, 64, 256, 129), (24, 1, 48, 32, 16, 15), (130, 1, 16, 16, 16, 40), (4, 2, 160, 32, 16, 47), (2, 1, 40, 24, 16, 17), (8, 2, 128, 128, 16, None),
    (4, 4, 128, 128, 16, 131)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_attention_sees_its_window_and_its_sink(Hq, Hkv, D, Dv, block, window, dtype):
    if dtype == "fp32" and Hq * D > 1024:
        pytest.skip("the same kernel at a smaller size")
    check_planted_keys(Hq, Hkv, D, Dv, block, _DTYPES[dtype], "cuda", length=150 if Hq * D < 400 else 139, window=window, sink=Hq != 12, elem_gate=Hq != 14)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("Hq,Hkv,D,Dv,window", [(8, 2, 128, 128, 300), (6, 2, 96, 64, 1000), (4, 4, 64, 128, 127), (4, 4, 64, 64, 260)])
def test_windowed_attention_long_portions_and_splits(Hq, Hkv, D, Dv, window):
    torch.manual_seed(D + Dv)
    bs, plan = 16, [(700, 390), (1500, 257), (64, 64), (2, 2), (1030, 1029), (1400, 1), (3, 1), (window + 1, 1)]
    cache = PagedKVCache(1, Hkv, D, sum((n + bs - 1) // bs for n, _ in plan), len(plan), 1600, bs, v_head_dim=Dv)
    entries, ks, vs = [], [], []
    for s, (n, new) in enumerate(plan):
        cache.reserve(s, n)
        k = _rnd(n, Hkv, D) * torch.linspace(0.3, 2.0, n, device="cuda").view(n, 1, 1)
        k, v = k.bfloat16(), _rnd(n, Hkv, Dv, dtype=torch.bfloat16)
        cache.append(0, k, v, torch.arange(n, dtype=torch.int32, device="cuda"), torch.full((n,), s, dtype=torch.int32, device="cuda"))
        entries.append((s, [0] * new, n - new, []))
        ks.append(k), vs.append(v)
    batch = RaggedBatch(entries, "cuda")
    q, gate, sink = _rnd(batch.n_rows, Hq, D, dtype=torch.bfloat16), _rnd(batch.n_rows, Hq, Dv, dtype=torch.bfloat16), _rnd(Hq, std=2.0)
    out = cache.attend(0, q, batch, gate=gate, window=window, sink=sink)
    rows = [(int(batch.slots[i]), i, int(batch.positions[i]), 1) for i in range(batch.n_single)] + batch.spans
    for n_splits in (1, 3):
        out[:batch.n_single] = cache.decode(0, q[:batch.n_single], batch.visible[:batch.n_single], None, n_splits, batch.slots[:batch.n_single],
                                            gate[:batch.n_single], window=window, sink=sink)
        for slot, row, start, n in rows:
            want, _ = R.attention(q[row:row + n][None], ks[slot][None], vs[slot][None], True, D ** -0.5, start, window, sink)
            want = R.head_gate(want[0], gate[row:row + n]).float()
            assert (out[row:row + n].float() - want).abs().max().item() < 4e-2, (slot, n_splits)
    assert _native.device_status(0) == 0


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("rows,H,count", [(1, 8, 5), (3, 4104, 4100), (2, 9000, 9000), (700, 1032, 1029)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_rms_rows_kernel(rows, H, count, dtype):
    dt, tol = _DTYPES[dtype], 1e-5 if dtype == "fp32" else 2e-2
    x, w = _rnd(rows, H), _rnd(H)
    x[:, count:] = 0
    want = O.one_plus_norm(x[:, :count].double(), w[:count].double(), 1e-4)
    got = D.rms_rows(x, w, 1e-4, count=count, offset=1.0, out_dtype=dt)
    assert got.dtype == dt and torch.allclose(got[:, :count].double(), want, atol=tol, rtol=1e-2 if dtype == "bf16" else 1e-5) and not got[:, count:].any()
    ids = torch.randint(0, rows, (5,), device="cuda")
    assert torch.equal(D.rms_rows(x, w, 1e-4, count=count, offset=1.0, rows=ids, out_dtype=dt), got[ids])
    table = x.to(dt)
    gx, h = D.embedding_rms(ids, table, w, 1e-4, count=count, offset=1.0)
    assert torch.equal(gx, table[ids].float()) and h.dtype == dt
    terms, where = _rnd(3 * rows, H, dtype=dt), torch.randperm(3 * rows, device="cuda").view(rows, 3).int()
    total = x + terms[where.long()].float().sum(1)
    want = O.one_plus_norm(total.double(), w.double(), 1e-4) if count == H else None
    y = x.clone()
    got = D.rms_rows(y, w, 1e-4, count=count, offset=1.0, pending=(terms, where), update=True, out_dtype=dt)
    assert torch.allclose(y, total, atol=1e-5)
    if want is not None:
        assert torch.allclose(got.double(), want, atol=tol * 2, rtol=1e-2 if dtype == "bf16" else 1e-5)
    assert torch.equal(D.rms_rows(x, w, 1e-4, count=count, offset=1.0, pending=(terms, where), rows=ids, out_dtype=dt), got[ids])


@pytest.mark.parametrize("heads,kv,dim,true_dim,vdim,rot", [(4, 2, 64, 64, 32, 64), (3, 1, 144, 136, 16, 10), (32, 8, 128, 128, 128, 64), (1, 1, 16, 9, 16, 8)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
@pytest.mark.parametrize("own", [True, False])
def test_head_finish_kernel(heads, kv, dim, true_dim, vdim, rot, dtype, own):
    dt = _DTYPES[dtype]
    cache = PagedKVCache(1, kv, dim, 40, 3, 300, 16, "cuda", dt, v_head_dim=vdim)
    host = PagedKVCache(1, kv, dim, 40, 3, 300, 16, "cpu", dt, v_head_dim=vdim)
    entries = [(1, [0], 250, []), (2, [0] * 90, 33, [])]
    for c in (cache, host):
        c.reserve(1, 251), c.reserve(2, 123)
    N = heads * dim + (kv * (dim + vdim) if own else 0) + 8
    packed = _rnd(91, N, dtype=dt)
    wq, wk = _rnd(dim), _rnd(dim)
    for t in [packed[:, :heads * dim].unflatten(1, (heads, dim))] + ([packed[:, heads * dim:(heads + kv) * dim].unflatten(1, (kv, dim))] if own else []):
        t[..., true_dim:] = 0
    ref = packed.cpu().clone()
    table = RotarySpec(rot, 100.0).table(300)
    kw = dict(heads=heads, dim=dim, k_off=heads * dim, v_off=(heads + kv) * dim, own_keys=own, true_dim=true_dim, eps=1e-3)
    D.qkv_head_finish(packed, cache, 0, RaggedBatch(entries, "cuda"), q_weight=wq, k_weight=wk, table=table.cuda(), **kw)
    D.qkv_head_finish(ref, host, 0, RaggedBatch(entries, "cpu"), q_weight=wq.cpu(), k_weight=wk.cpu(), table=table, **kw)
    tol = dict(atol=2e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=2e-2, rtol=1e-2)
    assert torch.allclose(packed.cpu().float(), ref.float(), **tol)
    assert torch.allclose(cache.k[0].cpu().float(), host.k[0].float(), **tol) and torch.equal(cache.v[0].cpu(), host.v[0])
    assert bool(cache.k[0].any()) == own


# ------------------------------------------------------------------ recurrence
@pytest.mark.parametrize("blocks,n,taps", [(3, 8, 4), (1, 72, 2), (2, 264, 1), (16, 128, 4)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_recurrence_kernels_over_unequal_portions(blocks, n, taps, dtype):
    # convolution, gates and scan against 64-bit sequences of their own; slots hold other sequences' leftovers
    torch.manual_seed(n)
    dt, W = _DTYPES[dtype], blocks * n
    plans = {0: [1, 300, 1, 1, 2, 129], 2: [700], 3: [2, 2, 1, 1, 128, 1], 1: [1, 1, 1]}
    T = {s: sum(p) for s, p in plans.items()}
    zx, y = {s: _rnd(t, W, dtype=dt) for s, t in T.items()}, {s: _rnd(t, W, dtype=dt) for s, t in T.items()}
    cw, cb = _rnd(taps, W, std=0.5), _rnd(W, std=0.2)
    gates, rb, ib = _rnd(blocks, 2, n, n, std=n ** -0.5, dtype=dt), _rnd(W), _rnd(W)
    lam = torch.linspace(-9.0, 1.5, W, device="cuda")[torch.randperm(W, device="cuda")]
    decay = -8.0 * torch.nn.functional.softplus(lam)
    state, conv = torch.full((5, W), 3.0, device="cuda"), torch.full((5, taps - 1, W), 2.0, device="cuda", dtype=dt)
    got, at = {s: [] for s in plans}, dict.fromkeys(plans, 0)
    for step in range(6):
        entries = [(s, [0] * p[step], at[s], []) for s, p in plans.items() if step < len(p)]
        batch = RaggedBatch(entries, "cuda")
        order = [e for e in entries if len(e[1]) == 1] + [e for e in entries if len(e[1]) > 1]
        cx = torch.cat([zx[s][a:a + len(t)] for s, t, a, _ in order])
        yy = torch.cat([y[s][a:a + len(t)] for s, t, a, _ in order])
        u = D.causal_conv(cx, cw, cb, conv, batch)
        out = torch.full((batch.n_rows, W + 8), 7.0, device="cuda", dtype=dt)
        D.gated_recurrence(u, yy, gates, rb, ib, decay, state, batch, cx, conv, out[:, :W])
        assert bool((out[:, W:] == 7.0).all())
        row = 0
        for s, t, a, _ in order:
            got[s].append(out[row:row + len(t), :W])
            row += len(t)
            at[s] = a + len(t)
    for s in plans:
        u = O.causal_convolution(zx[s].double().cpu(), cw.t().double().cpu(), cb.double().cpu())
        r = torch.sigmoid(O.block_linear(u, gates[:, 0].double().cpu(), rb.double().cpu().view(blocks, n)))
        i = torch.sigmoid(O.block_linear(u, gates[:, 1].double().cpu(), ib.double().cpu().view(blocks, n)))
        want = O.gated_linear_recurrence(u, r, i, lam.double().cpu()) * O.gelu_tanh(y[s].double().cpu())
        err = (torch.cat(got[s]).double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert float(err.max()) < (2e-5 if dtype == "fp32" else 2e-2), s
    assert bool((state[4] == 3.0).all()) and _native.device_status(0) == 0


@pytest.mark.parametrize("bn", [64, 128, 256])
def test_gate_product_tile_widths(bn):
    torch.manual_seed(bn)
    blocks, n, T = 2, 200, 300
    W = blocks * n
    u, y = _rnd(T, W, dtype=torch.bfloat16), _rnd(T, W, dtype=torch.bfloat16)
    gates, rb, ib, decay = _rnd(blocks, 2, n, n, std=n ** -0.5, dtype=torch.bfloat16), _rnd(W), _rnd(W), -torch.rand(W, device="cuda")
    outs = []
    for b in (0, bn):
        state, out = torch.zeros(2, W, device="cuda"), torch.empty(T, W, device="cuda", dtype=torch.bfloat16)
        D.gated_recurrence(u, y, gates, rb, ib, decay, state, RaggedBatch([(1, [0] * T, 0, [])], "cuda"), u, torch.zeros(2, 0, W, device="cuda"), out, bn=b)
        outs.append((state, out))
    assert torch.equal(outs[0][1], outs[1][1]) and torch.equal(outs[0][0], outs[1][0])


def test_long_memory_is_exact_to_the_last_place():
    # decays of 1 - 1e-4 over thousands of tokens, in one portion and token by token
    W, T = 64, 3000
    u = torch.ones(T, W, device="cuda")
    decay = -torch.logspace(-5, -2, W, device="cuda")
    gates, zero = torch.zeros(1, 2, W, W, device="cuda"), torch.zeros(W, device="cuda")
    log_a = 0.5 * decay.double()
    want = torch.sqrt(-torch.expm1(2 * log_a)) * 0.5 * -torch.expm1(T * log_a) / -torch.expm1(log_a)
    y = torch.full((T, W), 20.0, device="cuda")
    for cut in (T, 250):
        state, at = torch.zeros(1, W, device="cuda"), 0
        while at < T:
            D.gated_recurrence(u[at:at + cut], y[at:at + cut], gates, zero, zero, decay, state, RaggedBatch([(0, [0] * cut, at, [])], "cuda"), u,
                               torch.zeros(1, 0, W, device="cuda"), torch.empty(cut, W, device="cuda"))
            at += cut
        assert float((state[0].double() / want - 1).abs().max()) < 1e-4


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,H,experts,top", [(1, 64, 5, 1), (70, 72, 8, 2), (600, 64, 40, 7), (33, 128, 3, 3), (1500, 256, 300, 4), (9, 2056, 16, 2)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_routing(T, H, experts, top, dtype):
    torch.manual_seed(T)
    dt = _DTYPES[dtype]
    h, router = _rnd(T, H, dtype=dt), _rnd((experts + 7) // 8 * 8, H, std=2 * H ** -0.5, dtype=dt)
    route = D.moe_route(h, router, experts, top)
    z = h.double() @ router[:experts].double().t()
    index, place = route.index.long(), route.place.long()
    best = z.topk(top, -1)
    assert float((z.gather(1, index) - best.values).abs().max()) < 1e-4       # the largest, up to ties of rounding
    assert torch.allclose(route.weight.double(), torch.sigmoid(z.gather(1, index)), atol=1e-5)
    assert all(len(set(r)) == top for r in index.tolist())
    assert sorted(place.flatten().tolist()) == list(range(T * top))
    assert torch.equal(route.sorted[place], h[:, None].expand(T, top, H)) and torch.equal(route.scale[place], route.weight)
    seen, n = [], int(route.n_items)
    for e, lo, rows in route.items[:n].tolist():
        assert 0 < rows <= 128
        seen += [(e, p) for p in range(lo, lo + rows)]
    assert sorted(seen) == sorted(zip(index.flatten().tolist(), place.flatten().tolist()))


def test_equal_logits_take_the_lower_expert():
    h, router = torch.ones(3, 64, device="cuda"), torch.ones(8, 64, device="cuda")
    router[0] = -1
    assert D.moe_route(h, router, 5, 3).index.tolist() == [[1, 2, 3]] * 3
    h = torch.ones(600, 64, device="cuda")
    assert D.moe_route(h, router, 5, 3).index.tolist() == [[1, 2, 3]] * 600


@pytest.mark.parametrize("T,H,ff,experts,top,bn", [(1, 64, 24, 5, 2, 0), (20, 72, 40, 8, 2, 64), (300, 128, 136, 6, 2, 0), (300, 128, 136, 6, 2, 256), (900, 64, 264, 3, 1, 128),
                                                  (64, 1024, 520, 16, 2, 0), (2000, 256, 256, 4, 2, 0)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_grouped_products(T, H, ff, experts, top, bn, dtype):
    torch.manual_seed(T)
    dt = _DTYPES[dtype]
    h, router = _rnd(T, H, dtype=dt), _rnd((experts + 7) // 8 * 8, H, std=H ** -0.5, dtype=dt)
    gate_up, down = _rnd(experts, 2, ff, H, std=H ** -0.5, dtype=dt), _rnd(experts, 1, H, ff, std=ff ** -0.5, dtype=dt)
    route = D.moe_route(h, router, experts, top)
    act = D.grouped_linear(route.sorted, gate_up, route, glu="silu", seg_rows=T, bn=bn)
    y = D.grouped_linear(act, down, route, seg_rows=T, bn=bn)
    expert = torch.empty(T * top, dtype=torch.long, device="cuda")
    expert[route.place.long()] = route.index.long()
    tol = 1e-5 if dtype == "fp32" else 1e-2
    for e in range(experts):
        rows = expert == e
        s, x = route.scale[rows].double()[:, None], route.sorted[rows].double()
        want = O.silu(s * x @ gate_up[e, 0].double().t()) * (s * x @ gate_up[e, 1].double().t())
        assert torch.allclose(act[rows].double(), want, atol=tol, rtol=tol), e
        assert torch.allclose(y[rows].double(), act[rows].double() @ down[e, 0].double().t(), atol=tol, rtol=tol), e
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("M", [1, 60, 128, 129, 700])
def test_squared_relu_and_bias_in_the_product(M):
    for N, K in ((1032, 2056), (72, 64), (20008, 512)):
        a, w, b = _rnd(M, K, dtype=torch.bfloat16), _rnd(N, K, std=K ** -0.5, dtype=torch.bfloat16), _rnd(N)
        z = a.double() @ w.double().t() + b.double()
        assert torch.allclose(F.linear_rows(a, w, b, "relu2").double(), torch.relu(z) ** 2, atol=2e-2, rtol=1e-2)
        assert torch.allclose(F.linear_rows(a, w, b).double(), z, atol=2e-2, rtol=1e-2)


def test_model_with_wide_layers_matches_its_fp32_self():
    # sizes that take the CTA-pair, small-batch and wide grouped products, long portions, graphs
    from ferrotorch_b200.models.serving import PagedStepper
    from ferrotorch_b200.models.zolorax import ZoloraxConfig, ZoloraxForCausalLM

    cfg = ZoloraxConfig.pattern(2000, 1096, 6, 10, 2, 128, 1704, experts=4, top=4, window=200, width=1280, blocks=5)
    got = {}
    toks = torch.randint(0, 2000, (900,), generator=torch.Generator().manual_seed(5)).tolist()
    weights = ZoloraxForCausalLM(cfg, torch.float32, "cuda").random_(0.04).checkpoint_tensors()
    weights = {k: v.bfloat16().float() for k, v in weights.items()}
    for dtype in (torch.float32, torch.bfloat16):
        model = ZoloraxForCausalLM(cfg, dtype, "cuda")
        model.load_tensors(weights)
        st = PagedStepper(model, 64, 16, 4, 1000, cuda_graph=dtype == torch.bfloat16)
        s = st.admit()
        rows = [st.feed([(s, toks[:810], [0, 127, 128, 199, 200, 809])])]
        rows += [st.feed([(s, toks[810 + 6 * i:816 + 6 * i], range(6))]) for i in range(5)]
        rows += [st.feed([(s, [t], [0])]) for t in toks[840:]]
        got[dtype] = torch.cat(rows).double()
    a, b = got[torch.float32], got[torch.bfloat16]
    err = (a - b).pow(2).mean(-1).sqrt() / a.pow(2).mean().sqrt()
    assert float(err.max()) < 0.03 and _native.device_status(0) == 0

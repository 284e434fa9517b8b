"""The Mogelix decoder on its kernels, bf16 and fp32, against the plain oracle; the kernels alone at larger sizes."""
import pytest
import torch

import decoder_cases as C
import mogelix_oracle as O
from mogelix_cases import CASES, Case
from ferrotorch_b200 import _native
from ferrotorch_b200.models.mogelix import MogelixConfig, MogelixForCausalLM
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.nn.recurrent import StateSpaceSpec, StateSpaceState
from ferrotorch_b200.ops import decoder as D
from ferrotorch_b200.ops import reference as R
from planted_blocks import check_planted_blocks

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
    assert _native.launch_count() - before >= 1 + 3 * len(case.cfg["layers"])


@pytest.mark.parametrize("block", [4, 8, 16, 64])
def test_portions_and_single_tokens(case, block):
    C.check_portions(case, block)


@pytest.mark.parametrize("graph", [False, True], ids=["eager", "graph"])
def test_unequal_requests_in_one_batch(case, graph):
    C.check_batches(case, cuda_graph=graph)


def test_long_prompts_and_long_decoding(case):
    toks = case.tokens(330, 71)
    want = case.oracle(toks)
    for cuts in ([330], [130, 129, 1, 1, 1, 60, 1], [200, 1]):
        case.check(C.feed_all(case, cuts, toks), want, "cuts %s" % cuts)


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


# ------------------------------------------------------------------ attention: window and pooled blocks
@pytest.mark.parametrize("Hq,Hkv,D_,Dv,block,window,pool", [
    (6, 2, 16, 48, 8, 20, 5), (4, 4, 64, 64, 16, 33, 16), (8, 2, 128, 128, 16, 10, 3), (8, 1, 64, 64, 32, 1, 1), (5, 1, 48, 80, 4, 50, 7), (12, 2, 112, 96, 64, 128, 12),
    (14, 2, 128, 64, 256, 129, 2), (24, 1, 48, 32, 16, 15, 4), (4, 2, 160, 32, 16, 47, 9), (3, 1, 64, 128, 16, 100, 64), (2, 2, 32, 16, 8, 3, 1)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_attention_sees_its_window_and_pooled_blocks(Hq, Hkv, D_, Dv, block, window, pool, dtype):
    if dtype == "fp32" and Hq * D_ > 1024:
        pytest.skip("the same kernel at a smaller size")
    check_planted_blocks(Hq, Hkv, D_, Dv, block, _DTYPES[dtype], "cuda", 150 if Hq * D_ < 400 else 139, window, pool, sink=Hq != 14)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("Hq,Hkv,D_,Dv,window,pool", [(8, 2, 128, 128, 300, 2), (6, 2, 96, 64, 64, 1), (4, 4, 64, 64, 257, 16), (8, 1, 48, 112, 100, 5)])
def test_pooled_attention_long_portions_and_splits(Hq, Hkv, D_, Dv, window, pool):
    # more than one tile of pooled blocks; portions that begin far behind the first window
    torch.manual_seed(D_ + Dv)
    bs, plan = 16, [(700, 390), (1500, 257), (64, 64), (2, 2), (1030, 1029), (1400, 1), (3, 1), (window + pool, 1), (window + pool - 1, 1)]
    cache = PagedKVCache(1, Hkv, D_, sum((n + bs - 1) // bs for n, _ in plan), len(plan), 1600, bs, v_head_dim=Dv)
    cache.keep_pooled(0, pool)
    entries, ks, vs = [], [], []
    for s, (n, new) in enumerate(plan):
        cache.reserve(s, n)
        k = _rnd(n, Hkv, D_, dtype=torch.bfloat16) + _rnd(n // pool + 1, Hkv, D_)[torch.arange(n, device="cuda") // pool].bfloat16()
        v = _rnd(n, Hkv, Dv, dtype=torch.bfloat16)
        fill = RaggedBatch([(s, [0] * n, 0, [])], "cuda")
        cache.append(0, k, v, fill.positions, fill.slots)
        cache.pool_blocks(0, fill)
        entries.append((s, [0] * new, n - new, []))
        ks.append(k), vs.append(v)
    batch = RaggedBatch(entries, "cuda")
    q, sink = _rnd(batch.n_rows, Hq, D_, dtype=torch.bfloat16), _rnd(Hq)
    out = cache.attend(0, q, batch, window=window, pool=pool, sink=sink)
    rows = [(int(batch.slots[i]), i, int(batch.positions[i]), 1) for i in range(batch.n_single)] + batch.spans
    for n_splits in (1, 3, 8):
        n1 = batch.n_single
        out[:n1] = cache.decode(0, q[:n1], batch.visible[:n1], None, n_splits, batch.slots[:n1], window=window, pool=pool, sink=sink)
        for slot, row, start, n in rows:
            nb = len(ks[slot]) // pool
            pooled = tuple(t[slot][:nb * pool].float().unflatten(0, (nb, pool)).mean(1)[None] for t in (ks, vs))
            want, _ = R.attention(q[row:row + n][None].float(), ks[slot][None].float(), vs[slot][None].float(), True, D_ ** -0.5, start, window, sink, pool=pool, pooled=pooled)
            assert (out[row:row + n].float() - want[0]).abs().max().item() < 5e-2, (slot, n_splits)
    assert _native.device_status(0) == 0


# ------------------------------------------------------------------ state-space heads
@pytest.mark.parametrize("H,G,N,P", [(2, 1, 32, 64), (4, 2, 128, 64), (3, 3, 20, 200), (4, 1, 64, 256), (2, 2, 144, 32), (6, 2, 72, 136), (1, 1, 128, 256), (8, 1, 16, 48)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
@pytest.mark.parametrize("fast", [-4.0, 2.5])
def test_state_kernels_over_unequal_portions(H, G, N, P, dtype, fast):
    # token by token and in chunks against 64-bit sequences of their own; slots hold other sequences' leftovers; long and short memories
    torch.manual_seed(N + P)
    dt = _DTYPES[dtype]
    spec = StateSpaceSpec(H, P, N, G, 1)
    np_, vp = spec.padded_state, spec.padded_vdim
    plans = {0: [1, 300, 1, 1, 2, 129], 2: [700], 3: [2, 2, 1, 1, 128, 1], 1: [1, 1, 1, 257]}
    T = {s: sum(p) for s, p in plans.items()}

    def heads(t, n, d, padded):
        out = torch.zeros(t, n, padded, device="cuda", dtype=dt)
        out[:, :, :d] = _rnd(t, n, d, dtype=dt)
        return out.flatten(1)

    rows = {s: torch.cat([heads(t, H, P, vp), heads(t, G, N, np_), heads(t, G, N, np_)], 1) for s, t in T.items()}
    gates = {s: heads(t, H, P, vp) for s, t in T.items()}
    z = {s: torch.nn.functional.pad(_rnd(t, H, std=2.0), (0, 3)) for s, t in T.items()}
    bias, rate, skip = _rnd(H) - 1.0, torch.exp(_rnd(H) + fast), _rnd(H)
    want = {}
    for s, t in T.items():
        x, B, Cm = (c.double().cpu().view(t, n, -1) for c, n in zip(rows[s].split([H * vp, G * np_, G * np_], 1), (H, G, G)))
        step = O.softplus(z[s][:, :H].double().cpu() + bias.double().cpu())
        o = torch.stack([O.state_space(x[:, a], B[:, a // (H // G)], Cm[:, a // (H // G)], step[:, a], rate[a].double().cpu(), skip[a].double().cpu()) for a in range(H)], 1)
        want[s] = o * O.silu(gates[s].double().cpu().view(t, H, vp))
    for chunks in (False, True):
        state = torch.full((5, H, np_, vp), 3.0, device="cuda")
        got, at = {s: [] for s in plans}, dict.fromkeys(plans, 0)
        for step in range(6):
            entries = [(s, [0] * p[step], at[s], []) for s, p in plans.items() if step < len(p)]
            if not entries:
                continue
            batch = RaggedBatch(entries, "cuda")
            order = [e for e in entries if len(e[1]) == 1] + [e for e in entries if len(e[1]) > 1]
            u, zz, gg = (torch.cat([src[s][a:a + len(t)] for s, t, a, _ in order]) for src in (rows, z, gates))
            wide = torch.cat([gg, torch.ones_like(gg[:, :8])], 1)          # the gate lies in wider rows
            out = torch.full((batch.n_rows, H * vp + 8), 7.0, device="cuda", dtype=dt)
            D.state_space(u, wide[:, :H * vp], zz, bias, rate, skip, state, batch, out[:, :H * vp], heads=H, groups=G, chunks=chunks)
            assert bool((out[:, H * vp:] == 7.0).all())
            row = 0
            for s, t, a, _ in order:
                got[s].append(out[row:row + len(t), :H * vp])
                row += len(t)
                at[s] = a + len(t)
        for s in plans:
            o = torch.cat(got[s]).double().cpu().view(-1, H, vp)
            assert not o[..., P:].any()
            size = want[s].pow(2).mean((1, 2)).sqrt()     # of a row; results are rounded relative to their size
            err = (o - want[s]).pow(2).mean((1, 2)).sqrt() / (size + size.pow(2).mean().sqrt())
            assert float(err.max()) < (1e-5 if dtype == "fp32" else 8e-3), (s, chunks, int(err.argmax()))
        assert bool((state[4] == 3.0).all())
    assert _native.device_status(0) == 0


def test_state_is_the_same_in_chunks_and_token_by_token():
    torch.manual_seed(0)
    H, G, N, P, T = 4, 2, 128, 64, 1000
    u, gate = _rnd(T, H * P + 2 * G * N, dtype=torch.bfloat16), _rnd(T, H * P, dtype=torch.bfloat16)
    z, rate = _rnd(T, 8), torch.tensor([0.002, 0.05, 1.0, 16.0], device="cuda")
    states = []
    for cuts in ([T], [129, 871], [5] * 200):
        st, at = torch.zeros(1, H, N, P, device="cuda"), 0
        for n in cuts:
            r = slice(at, at + n)
            D.state_space(u[r], gate[r], z[r], torch.zeros(H, device="cuda"), rate, torch.ones(H, device="cuda"), st, RaggedBatch([(0, [0] * n, at, [])], "cuda"),
                          torch.empty(n, H * P, device="cuda", dtype=torch.bfloat16), heads=H, groups=G)
            at += n
        states.append(st)
    for st in states[:2]:
        assert float((st - states[2]).pow(2).mean((0, 2, 3)).sqrt().div(states[2].pow(2).mean((0, 2, 3)).sqrt()).max()) < 3e-4
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_convolution_with_silu_and_its_tail(taps, dtype):
    torch.manual_seed(taps)
    dt, Cn = _DTYPES[dtype], 1544
    x = {s: _rnd(150, Cn + 8, dtype=dt) for s in (0, 2)}
    w, b = _rnd(taps, Cn), _rnd(Cn)
    want = {s: O.silu(O.causal_conv(t[:, :Cn].double().cpu(), w.t().double().cpu(), b.double().cpu())) for s, t in x.items()}
    state, at = torch.full((4, taps - 1, Cn), 9.0, device="cuda", dtype=dt), {0: 0, 2: 0}
    for step in ({0: 1, 2: 37}, {0: 1}, {2: 2, 0: 2}, {0: 40, 2: 1}, {0: 1, 2: 3}, {2: 90, 0: 17}):
        entries = sorted(((s, [0] * n, at[s], []) for s, n in step.items()), key=lambda e: len(e[1]) > 1)
        batch = RaggedBatch(entries, "cuda")
        rows = torch.cat([x[s][a:a + len(t)] for s, t, a, _ in entries])[:, :Cn]
        u = D.causal_conv(rows, w, b, state, batch, silu=True)
        D.conv_tail(rows, state, batch)
        row = 0
        for s, t, a, _ in entries:
            assert torch.allclose(u[row:row + len(t)].double().cpu(), want[s][a:a + len(t)], **(dict(atol=1e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=1e-2, rtol=1e-2)))
            row += len(t)
            at[s] = a + len(t)
    assert bool((state[[1, 3]] == 9.0).all())


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("rows,H,count", [(1, 8, 5), (70, 200, 196), (5, 4096, 4096), (300, 1032, 1029), (2, 16384, 16380), (3, 6144, 6144)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_sum_norm_kernel(rows, H, count, dtype):
    torch.manual_seed(H)
    dt, tol = _DTYPES[dtype], dict(atol=2e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=4e-2, rtol=1e-2)
    x, y, terms, table = _rnd(rows, H), _rnd(rows, H, dtype=dt), _rnd(11, H, dtype=dt), _rnd(13, H, dtype=dt)
    packed = _rnd(rows, H + 16, dtype=dt)
    gate, w, last = packed[:, 8:8 + H], _rnd(H), _rnd(H)
    for t in (x, y, terms, table):
        t[..., count:] = 0
    ids = torch.randint(0, 13, (rows,), device="cuda")
    where, weight, dw = torch.randint(0, 11, (rows, 6), device="cuda").int(), torch.rand(rows, 6, device="cuda"), torch.rand(rows, device="cuda")
    for sub in (D.SublayerTerms(dense=y), D.SublayerTerms(terms, where, weight, y, dense_weight=dw), D.SublayerTerms(terms, where[:, :2].contiguous(), weight[:, :2].contiguous())):
        for g in (gate, None):
            total = sub.total().double() * (torch.sigmoid(g.double()) if g is not None else 1.0)
            for src, at in ((x, None), (table, ids)):
                s = 1.7 * (x if at is None else table[ids]).double() + total
                want = s / torch.sqrt(s.pow(2).sum(-1, keepdim=True) / count + 1e-3) * w.double()
                kw = dict(count=count, out_dtype=dt, ids=at)
                pick = torch.randint(0, rows, (4,), device="cuda")
                end = want / torch.sqrt(want.pow(2).sum(-1, keepdim=True) / count + 1e-3) * last.double()
                kept, part = D.sum_norm(src, sub, g, 1.7, w, 1e-3, rows=pick, last=last, **kw)
                assert kept is None and part.dtype == dt and torch.allclose(part.double(), end[pick], **tol)
                gx, gh = D.sum_norm(src.clone(), sub, g, 1.7, w, 1e-3, **kw)
                assert gx.dtype == torch.float32 and gh.dtype == dt and torch.allclose(gx.double(), want, atol=2e-5, rtol=1e-5) and torch.allclose(gh.double(), want, **tol)
                assert (gx.data_ptr() == gh.data_ptr()) == (dtype == "fp32")
                _, two = D.sum_norm(src.clone(), sub, g, 1.7, w, 1e-3, last=last, **kw)
                assert torch.allclose(two.double(), end, **tol)


@pytest.mark.parametrize("rows,heads,vdim,vp,parts", [(1, 3, 20, 32, 4), (70, 8, 64, 64, 1), (5, 128, 64, 64, 8), (300, 6, 16, 16, 3), (3, 200, 64, 64, 1), (9, 48, 128, 128, 48),
                                                     (4, 5, 33, 48, 15), (2, 96, 128, 128, 2)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_part_norm_kernel(rows, heads, vdim, vp, parts, dtype):
    torch.manual_seed(heads)
    dt = _DTYPES[dtype]
    y, w = torch.zeros(rows, heads, vp, device="cuda", dtype=dt), torch.zeros(heads, vp, device="cuda")
    y[..., :vdim], w[:, :vdim] = _rnd(rows, heads, vdim, dtype=dt), _rnd(heads, vdim)
    want = O.parts_rms(y[..., :vdim].flatten(1).double(), parts, 1e-3) * w[:, :vdim].flatten().double()
    buf = torch.cat([y.flatten(1), torch.full((rows, 8), 7.0, device="cuda", dtype=dt)], 1)
    D.part_norm_(buf[:, :heads * vp], w.flatten(), parts, 1e-3, heads=heads, vdim=vdim)
    got = buf[:, :heads * vp].view(rows, heads, vp)
    assert torch.allclose(got[..., :vdim].flatten(1).double(), want, **(dict(atol=1e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=2e-2, rtol=1e-2)))
    assert not got[..., vdim:].any() and bool((buf[:, heads * vp:] == 7.0).all())


@pytest.mark.parametrize("rows,N,count", [(1, 8, 3), (70, 200, 197), (5, 4096, 4096), (300, 8192, 8190), (3, 21504, 21504), (2, 30008, 30001)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_poly_norm_kernel(rows, N, count, dtype):
    torch.manual_seed(N)
    dt = _DTYPES[dtype]
    packed, coef = _rnd(rows, N + 24, dtype=dt), torch.tensor([0.7, -0.4, 0.9, 0.25], device="cuda")
    z = packed[:, :N]
    z[:, count:] = 0
    got = D.poly_norm(z, coef, 1e-3, count=count)
    want = O.poly_norm(z[:, :count].double(), *coef.double().tolist(), 1e-3)
    assert torch.allclose(got[:, :count].double(), want, **(dict(atol=3e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=2e-2, rtol=1e-2)))
    assert torch.allclose(got[:, count:].double(), coef[3].double().expand(rows, N - count), atol=2e-3)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,H,experts,top", [(1, 64, 5, 2), (70, 72, 8, 3), (600, 64, 40, 7), (33, 128, 2, 2), (1500, 256, 300, 4), (9, 2056, 16, 3)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_routing_with_bias_and_gate_and_experts_without_a_gate(T, H, experts, top, dtype):
    torch.manual_seed(T)
    dt, ff = _DTYPES[dtype], 40
    h, router, bias = _rnd(T, H, dtype=dt), _rnd((experts + 8) // 8 * 8, H, std=2 * H ** -0.5, dtype=dt), _rnd(experts)
    route = D.moe_route(h, router, experts, top, score="softmax", normalize=True, bias=bias, gate=True)
    z = h.double() @ router[:experts].double().t() + bias.double()
    index, place = route.index.long(), route.place.long()
    assert float((z.gather(1, index) - z.topk(top, -1).values).abs().max()) < 1e-4
    assert torch.allclose(route.weight.double(), torch.softmax(z.gather(1, index), -1), atol=1e-5)
    assert torch.allclose(route.gate.double(), torch.sigmoid(h.double() @ router[experts].double()), atol=1e-5)
    assert all(len(set(r)) == top for r in index.tolist()) and sorted(place.flatten().tolist()) == list(range(T * top))
    w = _rnd(experts, 1, ff, H, std=H ** -0.5, dtype=dt)
    got = D.grouped_linear(route.sorted, w, route, seg_rows=T, activation="relu2")[place].double()
    up = torch.relu(torch.einsum("th,tjfh->tjf", h.double(), w[index, 0].double())) ** 2 if T * top * ff * H < 2e7 else None
    if up is not None:
        assert torch.allclose(got, up, **(dict(atol=1e-4, rtol=1e-4) if dtype == "fp32" else dict(atol=3e-2, rtol=2e-2)))
    plain = D.grouped_linear(route.sorted, w, route, seg_rows=T)[place].double()
    assert torch.allclose(got, torch.relu(plain) ** 2, atol=6e-2, rtol=2e-2)
    assert _native.device_status(0) == 0


def test_model_with_wide_layers_matches_its_fp32_self():
    # sizes that take the CTA-pair, small-batch and wide grouped products, long portions, more than one tile of blocks, graphs
    from ferrotorch_b200.models.serving import PagedStepper

    cfg = MogelixConfig.pattern(2000, 1096, 6, 10, 2, 128, 1704, window=100, pool=3, state_heads=24, state_dim=64, state=128, groups=3, experts=4, top=4, expert_ff=520,
                                shared_ff=1704, alpha=2.0)
    got = {}
    toks = torch.randint(0, 2000, (900,), generator=torch.Generator().manual_seed(5)).tolist()
    weights = MogelixForCausalLM(cfg, torch.float32, "cuda").random_(0.04).checkpoint_tensors()
    weights = {k: v.bfloat16().float() for k, v in weights.items()}
    for k in weights:
        if k.endswith("dt_bias"):
            weights[k] = weights[k] - 3.0
        if k.endswith("mlp.act"):
            weights[k] = weights[k] + 0.5
    for dtype in (torch.float32, torch.bfloat16):
        model = MogelixForCausalLM(cfg, dtype, "cuda")
        model.load_tensors(weights)
        st = PagedStepper(model, 64, 16, 4, 1000, cuda_graph=dtype == torch.bfloat16)
        s = st.admit()
        rows = [st.feed([(s, toks[:810], [0, 99, 100, 127, 128, 809])])]
        rows += [st.feed([(s, toks[810 + 6 * i:816 + 6 * i], range(6))]) for i in range(5)]
        rows += [st.feed([(s, [t], [0])]) for t in toks[840:]]
        got[dtype] = torch.cat(rows).double()
    a, b = got[torch.float32], got[torch.bfloat16]
    err = (a - b).pow(2).mean(-1).sqrt() / a.pow(2).mean().sqrt()
    assert float(err.max()) < 0.03 and _native.device_status(0) == 0

"""The Tenalorn decoder on its kernels, bf16 and fp32, against the plain oracle; the kernels alone at larger sizes."""
import pytest
import torch

import decoder_cases as C
import tenalorn_oracle as O
from tenalorn_cases import CASES, Case
from ferrotorch_b200 import _native
from ferrotorch_b200.models.tenalorn import BigramSpec, TenalornConfig, TenalornForCausalLM
from ferrotorch_b200.nn.latent_attention import LatentAttention, LatentSpec
from ferrotorch_b200.nn.packed_block import RotarySpec, head_slopes
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.nn.recurrent import MatrixMemorySpec, MatrixMemoryState
from ferrotorch_b200.ops import decoder as D
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
    assert _native.launch_count() - before >= 2 + 5 * len(case.cfg["layers"])


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


# ------------------------------------------------------------------ attention: chunks, distance bias, latent rows
@pytest.mark.parametrize("Hq,Hkv,D_,Dv,block,chunk", [
    (6, 2, 16, 48, 8, 20), (4, 4, 64, 64, 16, 33), (8, 2, 128, 128, 16, 64), (8, 1, 64, 64, 32, 1), (5, 1, 48, 80, 4, 50), (12, 2, 112, 96, 64, 128),
    (14, 2, 128, 64, 256, 129), (24, 1, 48, 32, 16, 15), (4, 2, 160, 32, 16, 47), (8, 2, 128, 128, 16, None), (3, 1, 64, 64, 16, 100)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
@pytest.mark.parametrize("bias", [False, True])
def test_attention_sees_its_chunk_with_a_distance_bias(Hq, Hkv, D_, Dv, block, chunk, dtype, bias):
    if dtype == "fp32" and Hq * D_ > 1024:
        pytest.skip("the same kernel at a smaller size")
    check_planted_keys(Hq, Hkv, D_, Dv, block, _DTYPES[dtype], "cuda", length=150 if Hq * D_ < 400 else 139, chunk=chunk, out_scale=1.0 if bias else 0.6,
                       slopes=head_slopes(Hq) if bias else None, elem_gate=Hq != 14)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("Hq,Hkv,D_,Dv,chunk", [(8, 2, 128, 128, 300), (6, 2, 96, 64, 1000), (4, 4, 64, 64, 257)])
def test_chunked_attention_long_portions_and_splits(Hq, Hkv, D_, Dv, chunk):
    torch.manual_seed(D_ + Dv)
    bs, plan = 16, [(700, 390), (1500, 257), (64, 64), (2, 2), (1030, 1029), (1400, 1), (3, 1), (chunk + 1, 1), (chunk, 1)]
    cache = PagedKVCache(1, Hkv, D_, sum((n + bs - 1) // bs for n, _ in plan), len(plan), 1600, bs, v_head_dim=Dv)
    entries, ks, vs = [], [], []
    for s, (n, new) in enumerate(plan):
        cache.reserve(s, n)
        k, v = _rnd(n, Hkv, D_, dtype=torch.bfloat16), _rnd(n, Hkv, Dv, dtype=torch.bfloat16)
        cache.append(0, k, v, torch.arange(n, dtype=torch.int32, device="cuda"), torch.full((n,), s, dtype=torch.int32, device="cuda"))
        entries.append((s, [0] * new, n - new, []))
        ks.append(k), vs.append(v)
    batch = RaggedBatch(entries, "cuda")
    q, slopes = _rnd(batch.n_rows, Hq, D_, dtype=torch.bfloat16), head_slopes(Hq).cuda() * 0.05
    out = cache.attend(0, q, batch, chunk=chunk, slopes=slopes, out_scale=1.5)
    rows = [(int(batch.slots[i]), i, int(batch.positions[i]), 1) for i in range(batch.n_single)] + batch.spans
    for n_splits in (1, 3):
        n1 = batch.n_single
        out[:n1] = cache.decode(0, q[:n1], batch.visible[:n1], None, n_splits, batch.slots[:n1], chunk=chunk, slopes=slopes, out_scale=1.5)
        for slot, row, start, n in rows:
            want, _ = R.attention(q[row:row + n][None].float(), ks[slot][None].float(), vs[slot][None].float(), True, D_ ** -0.5, start, chunk=chunk, slopes=slopes)
            assert (out[row:row + n].float() - 1.5 * want[0]).abs().max().item() < 5e-2, (slot, n_splits)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("H,width,rank,block", [(4, 64, 48, 16), (16, 160, 128, 8), (17, 208, 192, 32), (32, 576, 512, 16), (40, 320, 256, 128), (5, 48, 48, 16), (3, 640, 512, 16),
                                                (2, 128, 16, 4)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_latent_rows_serve_as_keys_and_values(H, width, rank, block, dtype):
    if dtype == "fp32" and H > 16:
        pytest.skip("the same kernel at a smaller size")
    check_planted_keys(H, 1, width, rank, block, _DTYPES[dtype], "cuda", length=141, shared=True, tolerance=None if dtype == "fp32" else 5e-2)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("H,width,rank", [(32, 576, 512), (9, 96, 64), (64, 288, 256)])
def test_latent_decoding_over_long_contexts_and_splits(H, width, rank):
    torch.manual_seed(H)
    lens, bs = [1, 127, 128, 129, 1000, 2047, 700], 16
    cache = PagedKVCache(1, 1, width, 280, len(lens), 2048, bs, v_head_dim=rank, values_in_keys=[True])
    for s in range(len(lens)):
        cache.reserve(s, lens[s])
    cache.k[0].copy_(_rnd(*cache.k[0].shape) * 0.7)
    q = _rnd(len(lens), H, width, dtype=torch.bfloat16)
    visible = torch.tensor(lens, dtype=torch.int32, device="cuda")
    for n_splits in (0, 1, 2, 7, 16):
        out = cache.decode(0, q, visible, width ** -0.5, n_splits)
        for s, n in enumerate(lens):
            rows = cache.gather(0, s, n)[0][:, 0].float()
            p = torch.softmax(q[s].float() @ rows.t() * width ** -0.5, -1)
            want = p @ rows[:, :rank]
            assert (out[s].float() - want).abs().max().item() < 2e-2, (s, n_splits)
    assert _native.device_status(0) == 0


@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(8, 96, 32, 128, 512), (3, 20, 12, 40, 72), (16, 64, 32, 64, 256), (2, 130, 60, 144, 100)])
def test_latent_attention_forms_keys_or_absorbs_them(heads, dim, rot, vdim, rank):
    # the same portions through both paths, contexts that begin in earlier steps, and the oracle
    torch.manual_seed(rank)
    W, eps = 256, 1e-5
    spec = LatentSpec(heads, dim, rot, vdim, rank, (dim + rot) ** -0.5, RotarySpec(rot, 500.0, interleaved=True))
    module = LatentAttention(W, spec, eps).cuda()
    module.cast_(torch.bfloat16)
    sd = {n: (torch.randn(s) * (s[-1] ** -0.5 if len(s) > 1 else 1.0)).bfloat16().cuda() for n, s in module._shapes().items()}
    module.load(sd)
    plan = {0: [200, 1, 60], 1: [5, 300, 1], 2: [1, 17, 140]}
    T = {s: sum(p) for s, p in plan.items()}
    h = {s: _rnd(t, W, dtype=torch.bfloat16) for s, t in T.items()}
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": spec.scale, "rot": {"base": 500.0, "dims": rot}}
    for formed in (True, False):
        keep = module.key_proj
        if not formed:
            module.key_proj = None
        cache = PagedKVCache(1, 1, spec.row_size, 60, 3, 400, 16, "cuda", v_head_dim=spec.padded_rank, values_in_keys=[True])
        got, at = {s: [] for s in plan}, dict.fromkeys(plan, 0)
        for step in range(3):
            entries = [(s, [0] * p[step], at[s], []) for s, p in plan.items()]
            for s, t, a, _ in entries:
                cache.reserve(s, a + len(t))
            batch = RaggedBatch(entries, "cuda")
            order = [e for e in entries if len(e[1]) == 1] + [e for e in entries if len(e[1]) > 1]
            y = module(torch.cat([h[s][a:a + len(t)] for s, t, a, _ in order]), batch, cache, 0).dense
            row = 0
            for s, t, a, _ in order:
                got[s].append(y[row:row + len(t)])
                row += len(t)
                at[s] = a + len(t)
        module.key_proj = keep
        for s in plan:
            want = O.latent_attention(h[s].double().cpu(), {n: t.double().cpu() for n, t in sd.items()}, m, eps)
            err = (torch.cat(got[s]).double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
            assert float(err.max()) < 3e-2, (s, formed)
    assert _native.device_status(0) == 0


# ------------------------------------------------------------------ matrix memory
@pytest.mark.parametrize("H,dim,vdim,cap", [(2, 32, 64, 15.0), (3, 128, 128, 6.0), (1, 20, 200, 4.0), (4, 64, 256, 15.0), (2, 144, 32, 2.0), (2, 72, 136, 8.0), (1, 128, 256, 15.0)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
@pytest.mark.parametrize("remember", [1.0, 8.0])
def test_memory_kernels_over_unequal_portions(H, dim, vdim, cap, dtype, remember):
    # token by token and in chunks against 64-bit sequences of their own; slots hold other sequences' leftovers
    torch.manual_seed(dim + vdim)
    dt, eps = _DTYPES[dtype], 1e-5
    spec = MatrixMemorySpec(H, dim, vdim, cap)
    dp, vp, G = spec.padded_dim, spec.padded_vdim, (H + 3) // 4 * 4
    plans = {0: [1, 300, 1, 1, 2, 129], 2: [700], 3: [2, 2, 1, 1, 128, 1], 1: [1, 1, 1, 257]}
    T = {s: sum(p) for s, p in plans.items()}

    def heads(t, d, padded):
        out = torch.zeros(t, H, padded, device="cuda", dtype=dt)
        out[:, :, :d] = _rnd(t, H, d, dtype=dt)
        return out.flatten(1)

    rows = {s: torch.cat([heads(t, dim, dp), heads(t, dim, dp), heads(t, vdim, vp), heads(t, vdim, vp)], 1) for s, t in T.items()}
    z = {s: torch.zeros(t, 2 * G, device="cuda") for s, t in T.items()}
    for s, t in T.items():
        z[s][:, :H], z[s][:, G:G + H] = _rnd(t, H, std=2.0), _rnd(t, H, std=2.0)
    ib, fb, norm = _rnd(H), remember + _rnd(H), torch.zeros(H, vp, device="cuda")
    norm[:, :vdim] = _rnd(H, vdim)
    want = {}
    for s, t in T.items():
        parts = [c.double().cpu().view(t, H, -1) for c in rows[s].split([H * dp, H * dp, H * vp, H * vp], 1)]
        q, k, v, g = parts[0][..., :dim] * dim ** -0.5, parts[1][..., :dim], parts[2][..., :vdim], parts[3][..., :vdim]
        zi, zf = z[s][:, :H].double().cpu() + ib.double().cpu(), z[s][:, G:G + H].double().cpu() + fb.double().cpu()
        gi, gf = O.capped(zi, cap), O.log_sigmoid(O.capped(zf, cap))
        o = torch.stack([O.rms(O.matrix_memory(q[:, a], k[:, a], v[:, a], gi[:, a], gf[:, a]), eps) for a in range(H)], 1)
        want[s] = o * norm[:, :vdim].double().cpu() * torch.sigmoid(g) * 0.7
    for chunks in (False, True):
        state = MatrixMemoryState(5, spec, "cuda")
        for t in (state.S, state.n, state.m):
            t.fill_(3.0)
        got, at = {s: [] for s in plans}, dict.fromkeys(plans, 0)
        for step in range(6):
            entries = [(s, [0] * p[step], at[s], []) for s, p in plans.items() if step < len(p)]
            if not entries:
                continue
            batch = RaggedBatch(entries, "cuda")
            order = [e for e in entries if len(e[1]) == 1] + [e for e in entries if len(e[1]) > 1]
            packed = torch.cat([rows[s][a:a + len(t)] for s, t, a, _ in order])
            zz = torch.cat([z[s][a:a + len(t)] for s, t, a, _ in order])
            out = torch.full((batch.n_rows, H * vp + 8), 7.0, device="cuda", dtype=dt)
            q, k, v, g = packed.split([H * dp, H * dp, H * vp, H * vp], 1)
            D.matrix_memory(q, k, v, g, zz, ib, fb, norm.flatten(), state, batch, out[:, :H * vp], heads=H, dim=dim, vdim=vdim, cap=cap, eps=eps,
                            out_scale=0.7, chunks=chunks)
            assert bool((out[:, H * vp:] == 7.0).all())
            row = 0
            for s, t, a, _ in order:
                got[s].append(out[row:row + len(t), :H * vp])
                row += len(t)
                at[s] = a + len(t)
        for s in plans:
            o = torch.cat(got[s]).double().cpu().view(-1, H, vp)
            assert not o[..., vdim:].any()
            err = (o[..., :vdim] - want[s]).pow(2).mean((1, 2)).sqrt() / want[s].pow(2).mean().sqrt()
            assert float(err.max()) < (2e-4 if dtype == "fp32" else 2e-2), (s, chunks, int(err.argmax()))
        assert bool((state.S[4] == 3.0).all()) and bool((state.m[4] == 3.0).all())
    assert _native.device_status(0) == 0


def test_memory_state_is_the_same_in_chunks_and_token_by_token():
    torch.manual_seed(0)
    spec, T, H = MatrixMemorySpec(2, 64, 128, 15.0), 1000, 2
    packed = _rnd(T, H * 2 * (64 + 128), dtype=torch.bfloat16)
    q, k, v, g = packed.split([128, 128, 256, 256], 1)
    z = _rnd(T, 8)
    args = (z, torch.zeros(H, device="cuda"), torch.full((H,), 6.0, device="cuda"), torch.ones(256, device="cuda"))
    kw = dict(heads=H, dim=64, vdim=128, cap=15.0, eps=1e-5)
    states = []
    for cuts in ([T], [129, 871], [5] * 200):
        st, at = MatrixMemoryState(1, spec, "cuda"), 0
        for n in cuts:
            r = slice(at, at + n)
            D.matrix_memory(q[r], k[r], v[r], g[r], args[0][r], *args[1:], st, RaggedBatch([(0, [0] * n, at, [])], "cuda"),
                            torch.empty(n, 256, device="cuda", dtype=torch.bfloat16), **kw)
            at += n
        states.append(st)
    for st in states[:2]:
        for a, b in ((st.S, states[2].S), (st.n, states[2].n), (st.m, states[2].m)):
            assert float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()) < 3e-4
    assert _native.device_status(0) == 0


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("rows,S,H,count", [(1, 1, 8, 5), (70, 3, 200, 196), (5, 4, 4096, 4096), (300, 2, 1032, 1029), (3, 7, 64, 64), (2, 16, 520, 520), (2, 2, 16384, 16380)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_stream_step_kernel(rows, S, H, count, dtype):
    torch.manual_seed(H + S)
    dt, tol = _DTYPES[dtype], 2e-5 if dtype == "fp32" else 2e-2
    x, y, own, terms = _rnd(rows, S, H), _rnd(rows, H, dtype=dt), _rnd(rows, H, dtype=dt), _rnd(11, H, dtype=dt)
    for t in (x, y, own, terms):
        t[..., count:] = 0
    mix, out, into, w = _rnd(S, S), _rnd(S), _rnd(S), _rnd(H)
    where, weight = torch.randint(-1, 11, (rows, 3), device="cuda").int(), torch.rand(rows, 3, device="cuda")
    for sub in (D.SublayerTerms(dense=y), D.SublayerTerms(terms, where, weight, y, own), D.SublayerTerms(terms, where.clamp(min=0), weight)):
        total = sub.total().double()
        for xs in (x, x[:, :1].expand(-1, S, -1)):
            new = O.streams_out([xs[:, s].double() for s in range(S)], mix.double(), out.double(), total)
            u = O.streams_in(new, into.double())
            want = u / torch.sqrt(u.pow(2).sum(-1, keepdim=True) / count + 1e-3) * w.double()
            src = xs.clone() if xs is x or S == 1 else xs
            gx, gh = D.stream_step(src, sub, mix, out, into, w, 1e-3, count=count, out_dtype=dt)
            assert gh.dtype == dt and torch.allclose(gx.double(), torch.stack(new, 1), atol=1e-4, rtol=1e-5)
            assert torch.allclose(gh.double(), want, atol=tol * 4, rtol=1e-2 if dtype == "bf16" else 1e-4)
            ids = torch.randint(0, rows, (4,), device="cuda")
            src = xs.clone() if xs is x or S == 1 else xs
            same, part = D.stream_step(src, sub, mix, out, into, w, 1e-3, count=count, out_dtype=dt, rows=ids)
            assert torch.equal(part, gh[ids]) and torch.equal(same, xs)


@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_bigram_embedding_kernel(dtype):
    torch.manual_seed(3)
    dt, V, W, buckets = _DTYPES[dtype], 300, 1000, 77
    table, bigram = _rnd(V, W, dtype=dt), _rnd(buckets + 1, W, dtype=dt)
    cache = PagedKVCache(1, 1, 16, 40, 3, 200, 16, "cuda", dt)
    cache.keep_tokens()
    toks = {s: torch.randint(0, V, (100,)).tolist() for s in (0, 2)}
    emb = {"scale": 1.7, "bigram": {"buckets": buckets, "mul_prev": 1031, "mul_cur": 77777}}
    tables = {"embed": table.double().cpu(), "bigram": bigram.double().cpu()}
    want = {s: O.embedding(t, tables, emb) for s, t in toks.items()}
    into, w, at = torch.tensor([0.4, -2.0], device="cuda"), _rnd(W), {0: 0, 2: 0}
    for cuts in ({0: 1, 2: 17}, {0: 15, 2: 1}, {0: 1}, {2: 30, 0: 40}, {0: 2, 2: 2}):
        entries = [(s, toks[s][at[s]:at[s] + n], at[s], []) for s, n in cuts.items()]
        for s, t, a, _ in entries:
            cache.reserve(s, a + len(t))
        batch = RaggedBatch(entries, "cuda")
        x, h = D.embed_bigram(batch, cache, table, bigram, 1.7, 1031, 77777, into, w, 1e-4, count=W, out_dtype=dt)
        for i, (s, pos) in enumerate(zip(batch.slots.tolist(), batch.positions.tolist())):
            assert torch.allclose(x[i].double().cpu(), want[s][pos], atol=1e-5), (s, pos)
        ref = O.rms(x.double() * -1.6, 1e-4) * w.double()
        assert torch.allclose(h.double(), ref, atol=1e-4 if dtype == "fp32" else 4e-2, rtol=1e-4 if dtype == "fp32" else 1e-2)
        for s, n in cuts.items():
            at[s] += n


def test_softcap_kernel():
    z = _rnd(37, 1004, std=20.0)
    want = O.capped(z.double(), 15.0)
    assert torch.allclose(D.softcap_(z, 15.0).double(), want, atol=1e-5)


@pytest.mark.parametrize("heads,dim,rot,dims,rank", [(3, 12, 6, 6, 20), (32, 96, 32, 32, 512), (5, 16, 24, 16, 40)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_latent_finish_kernel(heads, dim, rot, dims, rank, dtype):
    torch.manual_seed(rank)
    dt = _DTYPES[dtype]
    spec = LatentSpec(heads, dim, rot, 16, rank, 1.0, RotarySpec(dims, 90.0, interleaved=True))
    caches = [PagedKVCache(1, 1, spec.row_size, 40, 3, 300, 16, d, dt, v_head_dim=spec.padded_rank, values_in_keys=[True]) for d in ("cuda", "cpu")]
    entries = [(1, [0], 250, []), (0, [0], 7, []), (2, [0] * 90, 33, [])]
    for c in caches:
        c.reserve(1, 251), c.reserve(0, 8), c.reserve(2, 123)
    qw = heads * spec.head_size
    packed = _rnd(92, qw + spec.row_size + 16, dtype=dt)
    packed[:, qw + rank:qw + spec.padded_rank] = 0
    ref = packed.cpu().clone()
    weight = torch.zeros(spec.padded_rank, device="cuda")
    weight[:rank] = _rnd(rank)
    table = spec.rotary.table(300)
    for n_lat in (2, 92):
        lat = [torch.zeros(n_lat, heads, spec.row_size, device=d, dtype=dt) for d in ("cuda", "cpu")]
        p, r = packed.clone(), ref.clone()
        for t, c, dev, ql in ((p, caches[0], "cuda", lat[0]), (r, caches[1], "cpu", lat[1])):
            D.latent_finish(t, c, 0, RaggedBatch(entries, dev), heads=heads, q_off=0, q_head=spec.head_size, q_rot=spec.padded_dim, c_off=qw, rank=rank,
                            rank_pad=spec.padded_rank, weight=weight.to(dev), eps=1e-3, table=table.to(dev), q_lat=ql)
        tol = dict(atol=2e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=3e-2, rtol=1e-2)
        assert torch.equal(p[:, qw:].cpu(), ref[:, qw:]) and torch.allclose(p[n_lat:, :qw].cpu().float(), r[n_lat:, :qw].float(), **tol)
        assert torch.allclose(lat[0].cpu().float(), lat[1].float(), **tol) and torch.allclose(caches[0].k[0].cpu().float(), caches[1].k[0].float(), **tol)


# ------------------------------------------------------------------ experts and products by blocks
@pytest.mark.parametrize("T,H,experts,identity,top", [(1, 64, 5, 1, 2), (70, 72, 8, 0, 2), (600, 64, 40, 9, 7), (33, 128, 2, 3, 4), (1500, 256, 300, 20, 4), (9, 2056, 16, 2, 3)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_routing_by_corrected_scores(T, H, experts, identity, top, dtype):
    torch.manual_seed(T)
    dt, n = _DTYPES[dtype], experts + identity
    h, router, corr = _rnd(T, H, dtype=dt), _rnd((n + 7) // 8 * 8, H, std=2 * H ** -0.5, dtype=dt), _rnd(n, std=0.02)
    route = D.moe_route(h, router, experts, top, identity=identity, score="softmax", correction=corr, normalize=True)
    s = torch.softmax(h.double() @ router[:n].double().t(), -1)
    index, place = route.index.long(), route.place
    choice = s + corr.double()
    assert float((choice.gather(1, index) - choice.topk(top, -1).values).abs().max()) < 1e-5
    chosen = s.gather(1, index)
    assert torch.allclose(route.weight.double(), chosen / chosen.sum(-1, keepdim=True), atol=1e-5)
    assert all(len(set(r)) == top for r in index.tolist())
    real = index < experts
    assert bool((place[~real] == -1).all()) and sorted(place[real].tolist()) == list(range(int(real.sum())))
    assert torch.equal(route.sorted[place[real].long()], h[:, None].expand(T, top, H)[real])
    seen = []
    for e, lo, rows in route.items[:int(route.n_items)].tolist():
        seen += [(e, p) for p in range(lo, lo + rows)]
    assert sorted(seen) == sorted(zip(index[real].tolist(), place[real].tolist()))


@pytest.mark.parametrize("T,G,K,N,a_col,out_col,bn", [(1, 3, 24, 48, 40, 64, 0), (64, 32, 96, 512, 128, 544, 0), (300, 5, 72, 40, 72, 40, 64), (130, 8, 512, 128, 512, 128, 128),
                                                      (20, 1, 64, 200, 64, 200, 256)])
@pytest.mark.parametrize("dtype", list(_DTYPES))
def test_products_by_blocks(T, G, K, N, a_col, out_col, bn, dtype):
    torch.manual_seed(T)
    dt = _DTYPES[dtype]
    a, w = _rnd(T, (G - 1) * a_col + K + 8, dtype=dt), _rnd(G, 1, N, K, std=K ** -0.5, dtype=dt)
    gate = _rnd(T, G * out_col, dtype=dt)
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == "fp32" else dict(atol=2e-2, rtol=1e-2)
    for g_ in (None, gate):
        out = torch.full((T, G * out_col), 7.0, device="cuda", dtype=dt)
        D.block_linear(a, w, out, a_col=a_col, out_col=out_col, gate=g_, bn=bn)
        for g in range(G):
            want = a[:, g * a_col:g * a_col + K].double() @ w[g, 0].double().t()
            if g_ is not None:
                want = want * torch.sigmoid(gate[:, g * out_col:g * out_col + N].double())
            assert torch.allclose(out[:, g * out_col:g * out_col + N].double(), want, **tol), g
            assert bool((out[:, g * out_col + N:(g + 1) * out_col] == 7.0).all())
    few = D.few_outputs(a[:, :K].contiguous(), w[0, 0, :9])
    assert few.dtype == torch.float32 and torch.allclose(few.double(), a[:, :K].double() @ w[0, 0, :9].double().t(), atol=1e-4)
    w2 = _rnd(1, 2, N, K, std=K ** -0.5, dtype=dt)
    out = D.block_linear(a[:, :K], w2, torch.empty(T, N, device="cuda", dtype=dt), glu="silu", bn=bn)
    z = a[:, :K].double()
    assert torch.allclose(out.double(), O.silu(z @ w2[0, 0].double().t()) * (z @ w2[0, 1].double().t()), **tol)
    assert _native.device_status(0) == 0


def test_model_with_wide_layers_matches_its_fp32_self():
    # sizes that take the CTA-pair, small-batch and wide grouped products, long portions, graphs
    from ferrotorch_b200.models.serving import PagedStepper

    cfg = TenalornConfig.pattern(2000, 1096, 3, 10, 2, 128, 520, chunk=200, memory_heads=3, memory_dim=128, memory_vdim=128, rank=512, rot_dim=32,
                                 experts=4, top=4, identity=0, shared_ff=1704, streams=3, bigram=BigramSpec(4099, 1031, 77))
    got = {}
    toks = torch.randint(0, 2000, (900,), generator=torch.Generator().manual_seed(5)).tolist()
    weights = TenalornForCausalLM(cfg, torch.float32, "cuda").random_(0.04).checkpoint_tensors()
    weights = {k: v.bfloat16().float() for k, v in weights.items()}
    for k in weights:
        if k.endswith("f.b"):
            weights[k] = weights[k] + 4.0
    for dtype in (torch.float32, torch.bfloat16):
        model = TenalornForCausalLM(cfg, dtype, "cuda")
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

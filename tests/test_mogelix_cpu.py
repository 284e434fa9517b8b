"""The Mogelix decoder on the CPU path: every mechanism and the serving machinery around it against the plain oracle."""
import io
import json
import math

import pytest
import torch

import decoder_cases as C
import mogelix_oracle as O
from mogelix_cases import CASES, Case, config_dict, random_weights
from ferrotorch_b200.models import registry
from ferrotorch_b200.models.generation import GenerationConfig, generate
from ferrotorch_b200.models.mogelix import MogelixConfig, MogelixForCausalLM
from ferrotorch_b200.models.serving import ContinuousBatcher
from ferrotorch_b200.nn.feed_forward import ExpertSpec, PackedMLP, RoutedExperts
from ferrotorch_b200.nn.gated_attention import GatedAttention
from ferrotorch_b200.nn.packed_block import AttentionSpec, RotarySpec, WavelengthScaling
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.nn.recurrent import StateSpaceBlock, StateSpaceSpec, StateSpaceState
from ferrotorch_b200.ops import decoder as D
from planted_blocks import check_planted_blocks


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request):
    return Case(request.param)


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _pad(t, n=4):
    return torch.nn.functional.pad(t, (0, n))


# ------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("alpha", [1.0, 0.3, 4.0])
def test_norm_comes_after_the_gated_sum(alpha):
    g, T, W = _gen(1), 7, 20
    x, y, gate, w, last = (torch.randn(T, W, generator=g) for _ in range(5))
    want = O.normed_sum(x.double(), y.double() * torch.sigmoid(gate.double()), alpha, w[0].double(), 1e-3)
    kw = dict(count=W, out_dtype=torch.float32)
    args = (_pad(x), D.SublayerTerms(dense=_pad(y)), _pad(gate), alpha, _pad(w[0]), 1e-3)
    got, h = D.sum_norm(*args, **kw)
    assert torch.allclose(got[:, :W].double(), want, atol=1e-5) and not got[:, W:].any() and torch.equal(got, h)
    rows = torch.tensor([6, 0, 2])
    _, h = D.sum_norm(*args, rows=rows, last=_pad(last[0]), **kw)
    assert torch.allclose(h[:, :W].double(), (O.rms(want, 1e-3) * last[0].double())[rows], atol=1e-5)
    # rows of a table, routed terms with weights, a weighted dense row, no gate
    table, ids = torch.randn(9, W, generator=g), torch.randint(0, 9, (T,), generator=g)
    terms, where, weight, dw = torch.randn(11, W, generator=g), torch.randint(0, 11, (T, 3), generator=g), torch.rand(T, 3, generator=g), torch.rand(T, generator=g)
    s = D.SublayerTerms(_pad(terms), where.int(), weight, _pad(y), dense_weight=dw)
    want = O.normed_sum(table[ids].double(), (dw[:, None] * y + (weight[..., None] * terms[where]).sum(1)).double(), alpha, w[0].double(), 1e-3)
    got, _ = D.sum_norm(_pad(table), s, None, alpha, _pad(w[0]), 1e-3, ids=ids, **kw)
    assert torch.allclose(got[:, :W].double(), want, atol=1e-5)
    with pytest.raises(ValueError):
        D.stream_step(x[:, None], s, torch.ones(1, 1), torch.ones(1), torch.ones(1), w[0], 1e-3, count=W, out_dtype=torch.float32)


def test_poly_norm_and_part_norm():
    g = _gen(2)
    z, coef = torch.randn(5, 19, generator=g) * 3, torch.tensor([0.7, -0.4, 1.3, 0.25])
    got = D.poly_norm(_pad(z, 5), coef, 1e-2, count=19)
    assert torch.allclose(got[:, :19].double(), O.poly_norm(z.double(), *coef.double(), 1e-2), atol=1e-5)
    assert torch.allclose(got[:, 19:], coef[3].expand(5, 5))
    one = O.poly_norm(torch.tensor([[2.0, -2.0]]).double(), 1.0, 10.0, 100.0, 0.5, 0.0)      # every power of +-2 is +-1 over its own mean square
    assert one.tolist() == [[111.5, -90.5 + 0.0]]
    for heads, vdim, parts in ((3, 20, 4), (4, 16, 1), (2, 6, 12), (5, 8, 5)):
        y, w = torch.randn(6, heads, vdim, generator=g), torch.randn(heads, vdim, generator=g)
        want = O.parts_rms(y.flatten(1).double(), parts, 1e-3) * w.flatten().double()
        buf = _pad(y, 12).flatten(1).contiguous()
        D.part_norm_(buf, _pad(w, 12).flatten(), parts, 1e-3, heads=heads, vdim=vdim)
        got = buf.view(6, heads, -1)
        assert torch.allclose(got[..., :vdim].flatten(1).double(), want, atol=1e-5) and not got[..., vdim:].any()


@pytest.mark.parametrize("taps", [1, 2, 3, 7])
def test_convolution_with_silu_over_portions(taps):
    g, T, n = _gen(taps), 30, 16
    x, w, b = torch.randn(T, n, generator=g), torch.randn(taps, n, generator=g), torch.randn(n, generator=g)
    want = O.silu(O.causal_conv(x.double(), w.t().double(), b.double()))
    state, at, got = torch.full((3, taps - 1, n), 9.0), 0, []
    for k in (2, 1, 1, 5, 2, 1, 12, 6):
        batch = RaggedBatch([(1, [0] * k, at, [])], "cpu")
        got.append(D.causal_conv(x[at:at + k], w, b, state, batch, silu=True))
        D.conv_tail(x[at:at + k], state, batch)
        at += k
    assert torch.allclose(torch.cat(got).double(), want, atol=1e-5) and bool((state[[0, 2]] == 9.0).all())


@pytest.mark.parametrize("heads,vdim,state,groups,conv,parts", [(1, 8, 16, 1, 4, 1), (6, 20, 12, 2, 3, 5), (4, 9, 33, 4, 1, 2), (6, 16, 5, 3, 2, 6)])
def test_state_space_mixer_over_portions_equals_the_oracle(heads, vdim, state, groups, conv, parts):
    g, T, W, eps = _gen(vdim), 45, 28, 1e-4
    spec = StateSpaceSpec(heads, vdim, state, groups, conv, parts)
    spec.validate()
    mixer = StateSpaceBlock(W, spec, eps, residual_gate=True)
    sd = {n: torch.randn(s, generator=g) * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in mixer._shapes().items()}
    sd["dt_bias"] -= 2.0
    mixer.load(sd)
    for n, t in mixer.unpack().items():
        assert torch.equal(t, sd[n]), n
    h = torch.randn(T, W, generator=g)
    m = {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": parts}
    W64 = {n: t.double() for n, t in sd.items()}
    want = O.ssd_mixer(h.double(), W64, m, eps)
    gates = h.double() @ W64["rg"].T + W64["rg.b"]
    st = StateSpaceState(3, spec, "cpu", torch.float32)
    st.S.fill_(7.0), st.conv.fill_(7.0)                   # leftovers of another sequence
    got, gate, at = [], [], 0
    for n in (1, 2, 17, 1, 1, 20, 3):
        y, z = mixer.terms(_pad(h[at:at + n]), RaggedBatch([(1, [0] * n, at, [])], "cpu"), st)
        got.append(y.dense), gate.append(z)
        at += n
    got, gate = torch.cat(got), torch.cat(gate)
    assert torch.allclose(got[:, :W].double(), want, atol=1e-4, rtol=1e-4) and not got[:, W:].any()
    assert torch.allclose(gate[:, :W].double(), gates, atol=1e-5) and not gate[:, W:].any()
    assert bool((st.S[0] == 7.0).all()) and bool((st.S[2] == 7.0).all()) and bool((st.conv[0] == 7.0).all())


def test_states_decay_by_their_step():
    one = torch.ones(3, 1).double()
    out = O.state_space(one, one, one, torch.tensor([0.5, 0.25, 2.0]).double(), torch.tensor(2.0).double(), torch.tensor(3.0).double())
    s1 = 0.5 * math.exp(-0.5) + 0.25
    assert out.flatten().tolist() == pytest.approx([3.5, 3 + s1, 3 + s1 * math.exp(-4.0) + 2.0])


def test_rotation_by_wavelength():
    # turns over the original length: more than `high` keep, fewer than `low` are divided, the middle is mixed
    rot = {"dims": 8, "base": 16.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 2.0 * math.pi * 5.0}}
    f = O.frequencies(rot).tolist()                       # unscaled: 1, 1/2, 1/4, 1/8, i.e. 5, 2.5, 1.25 and 0.625 turns
    assert f == pytest.approx([1.0, 0.5 * (0.5 + 0.5 / 4.0), (1 - 0.25 / 3) * 0.25 / 4 + 0.25 / 3 * 0.25, 0.125 / 4])
    spec = RotarySpec(8, 16.0, WavelengthScaling(4.0, 1.0, 4.0, 2.0 * math.pi * 5.0))
    table = spec.table(50).double()
    a = torch.outer(torch.arange(50).double(), torch.tensor(f).double())
    assert torch.allclose(table[..., 0], a.cos(), atol=1e-6) and torch.allclose(table[..., 1], a.sin(), atol=1e-6)
    z = torch.randn(11, generator=_gen(3)).double()
    got = O.rotate_halves(z, 7, rot)
    assert torch.equal(got[8:], z[8:]) and got[1].item() == pytest.approx((z[1] * math.cos(7 * f[1]) - z[5] * math.sin(7 * f[1])).item())
    assert O.frequencies({"dims": 4, "base": 9.0}).tolist() == pytest.approx([1.0, 1 / 3])


@pytest.mark.parametrize("window,pool", [(41, 11), (1, 1), (5, 16), (16, 4), (17, 3), (64, 7), (3, 50), (200, 8), (128, 16)])
@pytest.mark.parametrize("Hq,Hkv,D_,Dv", [(4, 2, 32, 16), (3, 1, 48, 40)])
def test_attention_sees_its_window_and_pooled_blocks(window, pool, Hq, Hkv, D_, Dv):
    check_planted_blocks(Hq, Hkv, D_, Dv, 16 if pool != 3 else 4, torch.float32, "cpu", 130, window, pool)


def test_window_and_block_edges_exactly():
    # equal keys: the softmax is an average over the visible values, which name keys and blocks
    bs, L, window, pool = 8, 50, 12, 5
    cache = PagedKVCache(1, 1, 16, 8, 1, 64, bs, "cpu", torch.float32, v_head_dim=64)
    cache.keep_pooled(0, pool)
    for cuts in ([L], [1] * L, [11, 2, 11, 1, 12, 13]):
        at = 0
        cache.free_sequence(0)
        for n in cuts:
            cache.reserve(0, at + n)
            batch = RaggedBatch([(0, [0] * n, at, [])], "cpu")
            cache.append(0, torch.ones(n, 1, 16), torch.eye(64)[at:at + n, None], batch.positions, batch.slots)
            cache.pool_blocks(0, batch)
            out = cache.attend(0, torch.ones(n, 1, 16), batch, 1.0, window=window, pool=pool)
            for i in range(n):
                p = at + i
                blocks = [b for b in range(L) if b * pool + pool - 1 <= p - window]
                assert len(blocks) == O.visible_blocks(p, window, pool)
                share = torch.zeros(64)
                share[max(0, p - window + 1):p + 1] = 1.0
                share[:len(blocks) * pool] += 1.0 / pool
                assert torch.allclose(out[i, 0], share / (min(p + 1, window) + len(blocks)), atol=1e-6)
            at += n
    with pytest.raises(ValueError):
        cache.attend(0, torch.ones(1, 1, 16), RaggedBatch([(0, [0], 3, [])], "cpu"), 1.0, window=window, pool=4)
    with pytest.raises(ValueError):
        cache.attend(0, torch.ones(1, 1, 16), RaggedBatch([(0, [0], 3, [])], "cpu"), 1.0, pool=pool)


@pytest.mark.parametrize("pool,block", [(1, 4), (3, 4), (4, 4), (5, 4), (16, 4), (7, 16), (16, 16), (48, 16)])
def test_blocks_lie_with_the_page_of_their_last_position(pool, block):
    cache = PagedKVCache(1, 1, 8, 40, 1, 128, block, "cpu", torch.float32)
    cache.keep_pooled(0, pool)
    cache.reserve(0, 120)
    b = torch.arange(120 // pool)
    page, at = cache._pooled_places(torch.zeros_like(b), b, pool)
    assert at.min() >= 0 and at.max() < cache.pooled[0, pool][0].shape[1] and len(set(zip(page.tolist(), at.tolist()))) == len(b)
    assert page.tolist() == [cache.pages_of(0)[(i * pool + pool - 1) // block] for i in b.tolist()]


@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 24, 40, (16, 30.0, WavelengthScaling(3.0, 1.5, 5.0, 40.0))), (3, 1, 16, 8, None), (2, 2, 32, 32, (32, 90.0, None))])
def test_attention_mixer_over_portions_and_a_reader_of_its_keys(heads, kv, dim, vdim, rot):
    g, T, W, eps = _gen(dim), 40, 30, 1e-4
    rotary = RotarySpec(*rot) if rot else None
    own = GatedAttention(W, AttentionSpec(heads, kv, dim, vdim, 0.3, window=9, pool=4, rotary=rotary), eps, gate=False, norm_weights=False, bias=True, residual_gate=True)
    reader = GatedAttention(W, AttentionSpec(2 * kv, kv, dim, vdim, 0.2, window=6, pool=3, rotary=rotary, kv_from=0), eps, gate=False, norm_weights=False, bias=True,
                            residual_gate=True)
    sds = []
    for module in (own, reader):
        sd = {n: torch.randn(s, generator=g) * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in module._shapes().items()}
        module.load(sd)
        for n, t in module.unpack().items():
            assert torch.equal(t, sd[n]), n
        sds.append({n: t.double() for n, t in sd.items()})
    assert "k" not in sds[1] and "v.b" not in sds[1] and "q.b" in sds[1]
    h = torch.randn(T, W, generator=g)
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 0.3, "mask": {"size": 9, "pool": 4}}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1], **({"scaling": dict(vars(rot[2]))} if rot[2] else {})}
    want, shared = O.attention_mixer(h.double(), sds[0], m, eps)
    want2, _ = O.attention_mixer(h.double(), sds[1], {**m, "heads": 2 * kv, "scale": 0.2, "mask": {"size": 6, "pool": 3}}, eps, shared)
    for cuts in ([T], [1] * T, [3, 1, 17, 1, 2, 16]):
        a = own.attn
        cache = PagedKVCache(1, kv, a.padded_dim, 12, 2, 64, 8, "cpu", torch.float32, v_head_dim=a.padded_vdim)
        cache.keep_pooled(0, 4), cache.keep_pooled(0, 3)
        got, got2, at = [], [], 0
        for n in cuts:
            cache.reserve(1, at + n)
            batch = RaggedBatch([(1, [0] * n, at, [])], "cpu")
            y, z = own.terms(_pad(h[at:at + n], 2), batch, cache, 0)
            assert torch.allclose(z[:, :W].double(), h[at:at + n].double() @ sds[0]["rg"].T + sds[0]["rg.b"], atol=1e-5)
            got.append(y.dense)
            got2.append(reader.terms(_pad(h[at:at + n], 2), batch, cache, 0)[0].dense)
            at += n
        assert torch.allclose(torch.cat(got)[:, :W].double(), want, atol=5e-5) and torch.allclose(torch.cat(got2)[:, :W].double(), want2, atol=5e-5)


@pytest.mark.parametrize("experts,top,shared", [(5, 1, 12), (5, 3, None), (3, 3, 1), (40, 7, 16)])
def test_routed_experts(experts, top, shared):
    g, W, ff, T = _gen(experts), 20, 12, 30
    spec = MogelixConfig.experts(experts, top, ff, shared)
    spec.validate()
    module = RoutedExperts(W, spec, "relu2", residual_gate=True)
    sd = {n: torch.randn(s, generator=g) * (2 * s[1] ** -0.5 if len(s) > 1 else 1.0) for n, s in module._shapes().items()}
    module.load(sd)
    h = torch.randn(T, W, generator=g)
    y, gate = module.terms(_pad(h))
    got = y.total()
    W64 = {k: v.double() for k, v in sd.items()}
    want = O.mixture(h.double(), W64, {"router": {"top": top}, "shared": shared})
    assert torch.allclose(got[:, :W].double(), want, atol=1e-4) and not got[:, W:].any()
    assert torch.allclose(gate[:, :W].double(), h.double() @ W64["rg"].T + W64["rg.b"], atol=1e-5)
    assert all(torch.equal(v, sd[k]) for k, v in module.unpack().items())


def test_router_bias_weighs_and_the_weights_sum_to_one():
    z, router = torch.tensor([[1.0, 0.0]]), torch.tensor([[2.0, 0], [1.0, 0], [0.0, 0], [0.5, 0]])
    route = D.moe_route(z, router, 3, 2, score="softmax", normalize=True, bias=torch.tensor([-5.0, 0.0, 3.0]), gate=True)
    assert route.index.tolist() == [[2, 1]] and route.weight[0].tolist() == pytest.approx([1 / (1 + math.exp(-2.0)), 1 / (1 + math.exp(2.0))])
    assert route.gate.tolist() == pytest.approx([1 / (1 + math.exp(-0.5))])
    assert [(e, round(w, 6)) for e, w in O.route([-3.0, 1.0, 3.0], 2)] == [(2, round(float(route.weight[0, 0]), 6)), (1, round(float(route.weight[0, 1]), 6))]


def test_dense_feed_forward_with_poly_norm():
    g, W, ff = _gen(5), 22, 37
    module = PackedMLP(W, ff, "poly_norm", 1e-3, residual_gate=True)
    sd = {n: torch.randn(s, generator=g) * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in module._shapes().items()}
    module.load(sd)
    assert all(torch.equal(v, sd[k]) for k, v in module.unpack().items())
    h = torch.randn(9, W, generator=g)
    y, gate = module.terms(_pad(h, 2))
    W64 = {k: v.double() for k, v in sd.items()}
    assert torch.allclose(y.dense[:, :W].double(), O.dense(h.double(), W64, 1e-3), atol=1e-5) and not y.dense[:, W:].any()
    assert torch.allclose(gate[:, :W].double(), h.double() @ W64["rg"].T + W64["rg.b"], atol=1e-5)


# ------------------------------------------------------------------ the model
def test_whole_prompt(case):
    C.check_whole_prompt(case)


@pytest.mark.parametrize("block", [4, 16])
def test_portions_and_single_tokens(case, block):
    C.check_portions(case, block)


def test_unequal_requests_in_one_batch(case):
    C.check_batches(case)


def test_residual_after_every_layer(case):
    toks = case.tokens(19, 9)
    _, want = O.forward(case.cfg, case.weights, toks, every_layer=True)
    st, seen = case.stepper(32), {}
    st.reserve(st.admit(), 19)
    z = case.model.paged_forward(RaggedBatch([(0, toks, 0, [18, 3])], "cpu"), st.cache, on_layer=lambda i, x: seen.update({i: x.clone()}))
    width = case.cfg["width"]
    assert sorted(seen) == list(range(len(want)))
    for i, w in enumerate(want):
        assert torch.allclose(seen[i][:, :width].double(), w, atol=2e-4, rtol=1e-4) and not seen[i][:, width:].any()
    case.check(z, case.oracle(toks)[[18, 3]], "logits beside the residual")


def test_greedy_generation_through_the_scheduler(case):
    C.check_generation(case)


def test_generation_with_preemption():
    b = C.check_generation(Case("mixed"), blocks=5)       # starved: sequences give way and are recomputed
    assert b.stats.preemptions > 0


def test_states_are_not_shared_or_wound_back_but_pages_with_their_blocks_are():
    case = Case("mixed")
    prompts = [case.tokens(26, 40) + case.tokens(n, 50 + n) for n in (3, 9, 1)]
    plain = ContinuousBatcher(case.model, 64, 8, 3, 64).generate(prompts, 6)
    shared = ContinuousBatcher(case.model, 64, 8, 1, 64, prefix_caching=True)
    assert shared.prefix is None and shared.generate(prompts, 6) == plain
    case = Case("attention")
    plain = ContinuousBatcher(case.model, 64, 8, 3, 64).generate(prompts, 6)
    shared = ContinuousBatcher(case.model, 64, 8, 1, 64, prefix_caching=True)
    assert shared.generate(prompts, 6) == plain and shared.stats.prefix_hit_tokens >= 2 * 24
    looked = ContinuousBatcher(case.model, 64, 8, 3, 64)
    reqs = [looked.submit(p, 6, lookahead=4) for p in prompts]
    looked.run()
    assert [r.output for r in reqs] == plain


def test_dense_entry_points(case):
    prompts = torch.tensor([case.tokens(11, 60), case.tokens(11, 61)])
    logits = case.model(prompts)
    for row, p in zip(logits, prompts.tolist()):
        case.check(row, case.oracle(p), "dense forward")
    out = generate(case.model, prompts, GenerationConfig.greedy(5))
    for row, p in zip(out.tolist(), prompts.tolist()):
        tokens, gap = C.greedy(case, p, 5)
        assert gap < 1e-3 or row == p + tokens


def test_long_decoding():
    case = Case("mixed")
    toks = case.tokens(200, 70)
    case.check(C.feed_all(case, [3, 1], toks), case.oracle(toks), "long decoding")


def test_far_tokens_reach_the_logits_only_where_the_design_lets_them():
    # one windowed layer: an early token is hidden once it has left the window, until its block is seen
    cfg = config_dict("attention")
    cfg["layers"] = cfg["layers"][:1]
    cfg["layers"][0]["mixer"]["mask"] = {"size": 4, "pool": 6}
    a = C.DecoderCase.tokens(None, 40, 3)
    b = [(a[0] + 1) % C.VOCAB] + a[1:]
    reach = {}
    for pool in (6, None):
        if pool is None:
            del cfg["layers"][0]["mixer"]["mask"]["pool"]
        model = MogelixForCausalLM(MogelixConfig.from_dict(cfg), torch.float32)
        model.load_tensors(random_weights(cfg, 1))
        far = (model(torch.tensor([a])) - model(torch.tensor([b]))).abs().amax(-1)[0]
        reach[pool] = (far > 1e-4).nonzero().flatten().tolist()
    assert reach[None] == [0, 1, 2, 3] and reach[6] == [0, 1, 2, 3] + list(range(9, 40))


# ------------------------------------------------------------------ configuration, weights, registry, programs
def test_configuration_reader():
    cfg = config_dict("mixed")
    c = MogelixConfig.from_dict(cfg)
    assert c.num_hidden_layers == 6 and c.alpha == 1.7 and c.layers[0].mlp == 67 and c.layers[2].mlp is None and c.layers[2].mixer.kv_from == 0
    assert c.layers[0].mixer.window == 9 and c.layers[0].mixer.pool == 4 and c.layers[3].mixer.rotary is None
    assert c.layers[0].mixer.rotary.scaling == WavelengthScaling(3.0, 1.5, 5.0, 40.0) and c.layers[2].mixer.rotary.scaling is None
    assert c.layers[1].mixer == StateSpaceSpec(6, 20, 12, 2, 3, 4)
    assert c.layers[1].mlp == ExpertSpec(5, 2, 20, "softmax", False, True, "output", 0, 33, False, True, True) and c.layers[3].mlp.shared_ff is None
    for name in CASES:
        d = config_dict(name)
        c = MogelixConfig.from_dict(d)
        assert MogelixConfig.from_dict(c.to_dict()) == c
        assert c.num_parameters() == sum(t.numel() for t in random_weights(d).values())
    for breakage in (lambda d: d.update(architecture="Other"), lambda d: d["layers"][0].update(type="linear"), lambda d: d["layers"][0]["mlp"].update(kind="glu"),
                     lambda d: d["layers"][0]["mixer"].update(heads=5), lambda d: d.update(layers=[]), lambda d: d["layers"][1]["mixer"].update(groups=4),
                     lambda d: d["layers"][1]["mixer"].update(norm_groups=7), lambda d: d["layers"][1]["mixer"].update(conv=0),
                     lambda d: d["layers"][0]["mixer"]["mask"].update(pool=0), lambda d: d["layers"][0]["mixer"]["mask"].pop("size"),
                     lambda d: d["layers"][2]["mixer"].update(kv_from=1), lambda d: d["layers"][2]["mixer"].update(kv_from=3), lambda d: d["layers"][2]["mixer"].update(vdim=8),
                     lambda d: d["layers"][1]["mlp"]["router"].update(top=6), lambda d: d["layers"][0]["mlp"].update(ff=0), lambda d: d["layers"][0]["mixer"]["rot"].update(dims=26)):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            MogelixConfig.from_dict(bad)


def test_weights_load_save_and_are_all_checked(tmp_path):
    case = Case("mixed")
    case.save(tmp_path / "m")
    model = registry.load_causal_lm(str(tmp_path / "m"), torch.float32)
    assert isinstance(model, MogelixForCausalLM) and registry.family_of(str(tmp_path / "m")).name == "mogelix"
    assert all(torch.equal(a, b) for a, b in zip(model.buffers(), case.model.buffers()))
    for name, t in model.checkpoint_tensors().items():
        assert torch.equal(t, case.weights[name].float()), name
    model.save_pretrained(str(tmp_path / "again"))
    back = registry.load_causal_lm(str(tmp_path / "again"), torch.float32)
    assert all(torch.equal(a, b) for a, b in zip(back.buffers(), model.buffers()))
    fresh = MogelixForCausalLM(case.model.config, torch.float32)
    for change in (lambda w: w.pop("l1.mix.A_log"), lambda w: w.update({"l2.norm2": w["l1.norm2"]}), lambda w: w.update({"l2.mix.k": w["l0.mix.k"]}),
                   lambda w: w.update({"l0.rg1": w["l0.rg1"][:, 1:]}), lambda w: w.pop("l1.mlp.e4.up"), lambda w: w.pop("l1.mlp.shared.sg"),
                   lambda w: w.update({"l0.mlp.act": w["l0.mlp.act"][:3]}), lambda w: w.pop("l0.mix.q.b")):
        bad = dict(case.weights)
        change(bad)
        with pytest.raises((KeyError, ValueError)):
            fresh.load_tensors(bad)


def test_registry_hub_and_tiny_model():
    from ferrotorch_b200 import hub

    assert "mogelix" in registry.list_causal_lms()
    info = hub.get_model_info("mogelix-3b")
    assert info.build().num_parameters() == info.num_parameters
    assert MogelixForCausalLM.tiny_random(torch.float32)(torch.tensor([[1, 2, 3]])).shape == (1, 3, 1000)


def test_cache_holds_pooled_blocks_and_states_per_slot():
    cache = Case("mixed").model.make_paged_cache(4, 16, 3, 64)
    assert len(cache.k) == 2 and sorted(cache.states) == [1, 4] and not cache.rewindable
    assert sorted(cache.pooled) == [(0, 1), (0, 4), (0, 5), (1, 20)]             # readers keep blocks of their own sizes of the same keys
    assert cache.pooled[0, 4][0].shape == (4, 4, 2, 32) and cache.pooled[0, 5][1].shape == (4, 4, 2, 48) and cache.pooled[1, 20][0].shape == (4, 1, 3, 16)
    assert cache.states[1].S.shape == (4, 6, 16, 32) and cache.states[1].conv.shape == (4, 2, 6 * 32 + 4 * 16)
    assert Case("attention").model.make_paged_cache(4, 16, 3, 64).rewindable


def test_trace_replay_reuses_slots(tmp_path, monkeypatch, capsys):
    from ferrotorch_b200.models import trace

    case = Case("mixed")
    case.save(tmp_path / "m")
    (tmp_path / "out").mkdir()
    a, b = case.tokens(40, 80), case.tokens(21, 81)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}, {"id": "a", "tokens": a[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": [18, 3]}, {"id": "a", "tokens": a[18:], "want": [21]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [20]}], "end": ["c", "a"]},
             {"step": 4, "entries": [{"id": "d", "tokens": a, "want": [39]}], "end": ["d"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert trace.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(5)]
    want = {0: [(a, 0), (a, 16)], 2: [(b, 20), (b, 5), (a, 39)], 3: [(b, 20)], 4: [(a, 39)]}
    for step, rows in want.items():
        data = (tmp_path / "out" / ("%d.f32" % step)).read_bytes()
        got = torch.frombuffer(bytearray(data), dtype=torch.float32).view(len(rows), C.VOCAB)
        case.check(got, torch.stack([case.oracle(t)[i] for t, i in rows]), "step %d" % step)


def test_server_command_line_serves_the_family(tmp_path):
    from ferrotorch_b200.models import server

    args = ["--device", "cpu", "--port", "0", "--kv-pages", "16", "--serve-seconds", "0.2"]
    assert server.main(["--tiny", "--family", "mogelix", *args]) == 0
    Case("mixed").save(tmp_path / "m")
    assert server.main(["--model", str(tmp_path / "m"), *args]) == 0


def test_the_decoder_kernel_set_holds_every_kernel_the_cache_and_the_row_kernels_call():
    import os
    import re

    from ferrotorch_b200 import _native
    from ferrotorch_b200.nn import paged

    text = "".join(open(os.path.join(_native.CSRC, n + ".cu")).read() for n in _native.KERNEL_SETS["decoder"])
    have = set(re.findall(r"FT_API[^;{(]*?\b(ft_\w+)\s*\(", text))
    need = {n for m in (paged, D) for n in re.findall(r"\.(ft_\w+)\(", open(m.__file__).read())}
    assert {"ft_pool_blocks", "ft_state_chunks", "ft_sum_norm_rows", "ft_poly_norm"} <= need <= have, need - have

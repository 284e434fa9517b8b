"""The Tenalorn decoder on the CPU path: every mechanism and the serving machinery around it against the plain oracle."""
import io
import json

import pytest
import torch

import decoder_cases as C
import tenalorn_oracle as O
from tenalorn_cases import CASES, Case, config_dict, random_weights
from ferrotorch_b200.models import registry
from ferrotorch_b200.models.generation import GenerationConfig, generate
from ferrotorch_b200.models.serving import ContinuousBatcher
from ferrotorch_b200.models.tenalorn import TenalornConfig, TenalornForCausalLM
from ferrotorch_b200.nn.feed_forward import ExpertSpec, RoutedExperts
from ferrotorch_b200.nn.latent_attention import LatentAttention, LatentSpec
from ferrotorch_b200.nn.packed_block import AttentionSpec, RotarySpec, head_slopes
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.nn.parallel_mixer import AttentionMemoryMixer
from ferrotorch_b200.nn.recurrent import MatrixMemorySpec, MatrixMemoryState
from ferrotorch_b200.ops import decoder as D
from planted_keys import check_planted_keys


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request):
    return Case(request.param)


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


# ------------------------------------------------------------------ mechanisms
def test_bigram_rows_look_at_the_previous_token_and_the_first_token_has_its_own():
    V, W, buckets = 50, 16, 23
    g = _gen(1)
    table, bigram = torch.randn(V, W, generator=g), torch.randn(buckets + 1, W, generator=g)
    cache = PagedKVCache(1, 1, 16, 8, 2, 64, 4, "cpu", torch.float32)
    cache.keep_tokens()
    toks, other = [3, 7, 7, 49, 0, 12, 5, 5, 1], [9, 8, 4]
    want = O.embedding(toks, {"embed": table.double(), "bigram": bigram.double()}, {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": 11, "mul_cur": 6}})
    into, norm, at, got = torch.tensor([0.5, 1.5, -3.0]), torch.ones(W), 0, []
    for n, foreign in ((1, []), (1, [9]), (4, []), (2, [8, 4]), (1, [])):        # the last entry begins a page; another sequence in between
        entries = [(0, toks[at:at + n], at, [])] + ([(1, foreign, 0 if len(foreign) == 1 else 1, [])] if foreign else [])
        for s, t, a, _ in entries:
            cache.reserve(s, a + len(t))
        batch = RaggedBatch(entries, "cpu")
        x, h = D.embed_bigram(batch, cache, table, bigram, 2.5, 11, 6, into, norm, 1e-4, count=W, out_dtype=torch.float32)
        rows = [i for i, s in enumerate(batch.slots.tolist()) if s == 0]
        got.append(x[rows])
        assert torch.allclose(h[rows].double(), O.rms(-1.0 * x[rows].double(), 1e-4), atol=1e-5)
        at += n
    assert torch.allclose(torch.cat(got).double(), want, atol=1e-5)
    assert O.bigram_row(None, 5, 11, 6, buckets) == buckets and O.bigram_row(0, 0, 11, 6, buckets) == 0
    assert [int(cache.token_pages[p, i]) for p in cache.pages_of(1) for i in range(4)][:3] == other


@pytest.mark.parametrize("S", [1, 2, 5])
def test_streams_change_at_once_from_the_old_ones(S):
    g, T, W = _gen(S), 7, 20
    pad = torch.nn.functional.pad
    x, y, mix = torch.randn(T, S, W, generator=g), torch.randn(T, W, generator=g), torch.randn(S, S, generator=g)
    out, into, w = torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(W, generator=g)
    new = O.streams_out([x[:, s].double() for s in range(S)], mix.double(), out.double(), y.double())
    u = O.streams_in(new, into.double())
    args = (mix, out, into, pad(w, (0, 4)), 1e-3)
    gx, gh = D.stream_step(pad(x, (0, 4)), D.SublayerTerms(dense=pad(y, (0, 4))), *args, count=W, out_dtype=torch.float32)
    assert torch.allclose(gx[:, :, :W].double(), torch.stack(new, 1), atol=1e-5) and not gx[:, :, W:].any()
    assert torch.allclose(gh[:, :W].double(), O.rms(u, 1e-3) * w.double(), atol=1e-4)
    rows = torch.tensor([6, 0])
    _, part = D.stream_step(pad(x, (0, 4)), D.SublayerTerms(dense=pad(y, (0, 4))), *args, count=W, out_dtype=torch.float32, rows=rows)
    assert torch.allclose(part, gh[rows], atol=1e-6)
    # terms of experts, some of which are the input itself
    terms, own = torch.randn(9, W, generator=g), torch.randn(T, W, generator=g)
    where, weight = torch.randint(-1, 9, (T, 3), generator=g).int(), torch.rand(T, 3, generator=g)
    t = D.SublayerTerms(terms, where, weight, y, own)
    want = y + sum(weight[:, j, None] * torch.where(where[:, j, None] < 0, own, terms[where[:, j].clamp(min=0).long()]) for j in range(3))
    assert torch.allclose(t.total(), want, atol=1e-5)


@pytest.mark.parametrize("chunk,slopes", [(1, True), (16, False), (17, True), (40, True), (64, False), (128, True), (None, True)])
@pytest.mark.parametrize("Hq,Hkv,D_,Dv", [(6, 2, 32, 16), (3, 1, 48, 40)])
def test_attention_sees_its_chunk_with_a_distance_bias(chunk, slopes, Hq, Hkv, D_, Dv):
    check_planted_keys(Hq, Hkv, D_, Dv, 16, torch.float32, "cpu", length=130, chunk=chunk, slopes=head_slopes(Hq) if slopes else None, out_scale=0.7)


def test_chunk_edges_exactly():
    # equal keys: the softmax is an average over the visible values, which names the visible keys
    bs, L, chunk = 8, 50, 12
    cache = PagedKVCache(1, 1, 16, 8, 1, 64, bs, "cpu", torch.float32, v_head_dim=64)
    cache.reserve(0, L)
    pos = torch.arange(L, dtype=torch.int32)
    cache.append(0, torch.ones(L, 1, 16), torch.eye(64)[:L, None], pos, torch.zeros(L, dtype=torch.int32))
    for cuts in ([L], [1] * L, [11, 2, 11, 1, 12, 13]):
        at = 0
        for n in cuts:
            out = cache.attend(0, torch.ones(n, 1, 16), RaggedBatch([(0, [0] * n, at, [])], "cpu"), 1.0, chunk=chunk)
            for i in range(n):
                seen = (out[i, 0] > 1e-6).nonzero().flatten().tolist()
                assert seen == list(range((at + i) // chunk * chunk, at + i + 1))
            at += n


def test_slopes():
    for H in (1, 3, 8, 12):
        assert head_slopes(H).tolist() == pytest.approx([O.head_slope(h, H) for h in range(H)])
    assert head_slopes(8).tolist() == [2.0 ** -(h + 1) for h in range(8)]


@pytest.mark.parametrize("H,dim,vdim,cap", [(1, 8, 16, 15.0), (3, 20, 12, 4.0), (2, 33, 40, 1.0)])
def test_matrix_memory_over_portions_equals_the_oracle(H, dim, vdim, cap):
    g, T, W, eps = _gen(dim), 45, 28, 1e-4
    spec = MatrixMemorySpec(H, dim, vdim, cap)
    mixer = AttentionMemoryMixer(W, AttentionSpec(2, 1, 16, 16, 0.2, chunk=8, distance_bias=True), spec, 0.6, 1.7, eps)
    sd = {n: torch.randn(s, generator=g) * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in mixer._shapes().items()}
    sd["right.f.b"] += 3.0
    mixer.load(sd)
    for n, t in mixer.unpack().items():
        assert torch.equal(t, sd[n]), n
    h = torch.randn(T, W, generator=g)
    m = {"left": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.2, "mask": {"size": 8}},
         "right": {"heads": H, "dim": dim, "vdim": vdim, "gate_cap": cap}, "left_scale": 0.6, "right_scale": 1.7}
    want = O.parallel_mixer(h.double(), {n: t.double() for n, t in sd.items()}, m, eps)
    cache = PagedKVCache(1, 1, 16, 12, 3, 64, 8, "cpu", torch.float32)
    state = MatrixMemoryState(3, spec, "cpu")
    for t in (state.S, state.n, state.m):
        t.fill_(7.0)                                      # leftovers of another sequence
    got, at = [], 0
    for n in (1, 2, 17, 1, 1, 20, 3):
        cache.reserve(1, at + n)
        y = mixer(torch.nn.functional.pad(h[at:at + n], (0, 4)), RaggedBatch([(1, [0] * n, at, [])], "cpu"), cache, 0, state)
        got.append(y.dense)
        at += n
    got = torch.cat(got)
    assert torch.allclose(got[:, :W].double(), want, atol=2e-4, rtol=1e-4) and not got[:, W:].any()
    assert bool((state.S[0] == 7.0).all()) and bool((state.m[2] == 7.0).all())


def test_running_maximum_starts_at_zero_and_floors_the_denominator():
    # strongly negative input gates: the maximum stays at zero and exp(-m) = 1 outweighs |n.q|
    q, k, v = torch.ones(1, 4).double(), torch.ones(1, 4).double(), torch.ones(1, 2).double()
    o = O.matrix_memory(q, k, v, torch.tensor([-10.0]).double(), torch.tensor([-1.0]).double())
    assert o[0, 0].item() == pytest.approx(4 * 2.718281828 ** -10 / (1 + 1e-6), rel=1e-6)


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,dims", [(5, 20, 6, 24, 36, 6), (2, 16, 16, 16, 32, 16), (3, 8, 12, 40, 17, 8)])
def test_latent_attention_over_portions_equals_the_oracle(heads, dim, rot, vdim, rank, dims):
    g, T, W, eps = _gen(rank), 40, 30, 1e-4
    spec = LatentSpec(heads, dim, rot, vdim, rank, 0.3, RotarySpec(dims, 70.0, interleaved=True))
    spec.validate()
    module = LatentAttention(W, spec, eps)
    sd = {n: torch.randn(s, generator=g) * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in module._shapes().items()}
    module.load(sd)
    for n, t in module.unpack().items():
        assert torch.equal(t, sd[n]), n
    h = torch.randn(T, W, generator=g)
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": 0.3, "rot": {"base": 70.0, "dims": dims}}
    want = O.latent_attention(h.double(), {n: t.double() for n, t in sd.items()}, m, eps)
    for cuts in ([T], [1] * T, [3, 1, 17, 1, 2, 16]):
        cache = PagedKVCache(1, 1, spec.row_size, 12, 2, 64, 8, "cpu", torch.float32, v_head_dim=spec.padded_rank, values_in_keys=[True])
        got, at = [], 0
        for n in cuts:
            cache.reserve(1, at + n)
            got.append(module(torch.nn.functional.pad(h[at:at + n], (0, 2)), RaggedBatch([(1, [0] * n, at, [])], "cpu"), cache, 0).dense)
            at += n
        got = torch.cat(got)
        assert torch.allclose(got[:, :W].double(), want, atol=5e-5) and not got[:, W:].any()
    with pytest.raises(ValueError):
        cache.append(0, torch.zeros(1, 1, spec.row_size), torch.zeros(1, 1, spec.padded_rank), torch.zeros(1, dtype=torch.int32))


def test_rotation_turns_neighbours():
    z = torch.tensor([1.0, 0.0, 0.0, 2.0, 5.0]).double()
    got = O.rotate_pairs(z, 3, 4, 100.0)
    a, b = torch.tensor(3.0).double(), torch.tensor(0.3).double()
    assert torch.allclose(got, torch.stack([a.cos(), a.sin(), -2 * b.sin(), 2 * b.cos(), torch.tensor(5.0).double()]))
    from ferrotorch_b200.ops import reference as R
    table = RotarySpec(4, 100.0, interleaved=True).table(8)
    assert torch.allclose(R.rotate_pairs(z.float()[None, None], table, torch.tensor([3]))[0, 0].double(), got, atol=1e-6)


@pytest.mark.parametrize("experts,top,identity,shared", [(5, 1, 2, 12), (5, 3, 0, 7), (3, 4, 1, None), (40, 7, 9, 16)])
def test_routed_experts(experts, top, identity, shared):
    g, W, ff, T = _gen(experts), 20, 12, 30
    spec = TenalornConfig.experts(experts, top, ff, identity, shared)
    spec.validate()
    module = RoutedExperts(W, spec)
    sd = {n: torch.randn(s, generator=g) * (2 * s[1] ** -0.5 if len(s) > 1 else 0.1) for n, s in module._shapes().items()}
    module.load(sd)
    h = torch.randn(T, W, generator=g)
    got = module(torch.nn.functional.pad(h, (0, 4))).total()
    W64 = {k: v.double() for k, v in sd.items()}
    if shared is None:
        W64.update({"shared.gate": torch.zeros(1, W).double(), "shared.up": torch.zeros(1, W).double(), "shared.down": torch.zeros(W, 1).double()})
    want = O.mixture(h.double(), W64, {"top": top, "experts": experts})
    assert torch.allclose(got[:, :W].double(), want, atol=2e-5) and not got[:, W:].any()
    assert all(torch.equal(v, sd[k]) for k, v in module.unpack().items())


def test_correction_chooses_but_does_not_weigh():
    z = torch.tensor([[1.0, 0.0]])
    router = torch.tensor([[2.0, 0], [1.0, 0], [0.0, 0]])
    s = torch.softmax(z @ router.T, -1)[0]
    route = D.moe_route(z, router, 2, 2, identity=1, score="softmax", correction=torch.tensor([-5.0, 0.0, 3.0]), normalize=True)
    assert route.index.tolist() == [[2, 1]] and route.place.tolist() == [[-1, 0]]
    assert torch.allclose(route.weight[0], torch.stack([s[2], s[1]]) / (s[1] + s[2]))


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
    case.model.paged_forward(RaggedBatch([(0, toks, 0, [])], "cpu"), st.cache, on_layer=lambda i, x: seen.update({i: x.clone()}))
    width = case.cfg["width"]
    assert sorted(seen) == list(range(len(want)))
    for i, w in enumerate(want):
        assert torch.allclose(seen[i][:, :width].double(), w, atol=2e-4, rtol=1e-4) and not seen[i][:, width:].any()


def test_greedy_generation_through_the_scheduler(case):
    C.check_generation(case)


def test_generation_with_preemption():
    b = C.check_generation(Case("mixed"), blocks=5)       # starved: sequences give way and are recomputed
    assert b.stats.preemptions > 0


def test_states_are_not_shared_or_wound_back():
    case = Case("mixed")
    prompts = [case.tokens(26, 40) + case.tokens(n, 50 + n) for n in (3, 9, 1)]
    plain = ContinuousBatcher(case.model, 64, 8, 3, 64).generate(prompts, 6)
    shared = ContinuousBatcher(case.model, 64, 8, 1, 64, prefix_caching=True)
    assert shared.prefix is None and shared.generate(prompts, 6) == plain
    # without memories, prefixes are shared (their pages hold the previous token too) and tokens can be taken back
    case = Case("latent")
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
    toks = case.tokens(260, 70)
    case.check(C.feed_all(case, [3, 1], toks), case.oracle(toks), "long decoding")


def test_far_tokens_reach_the_logits_only_where_the_design_lets_them():
    # chunks hide a changed early token from attention; memories and latents remember it
    a = C.DecoderCase.tokens(None, 40, 3)
    b = [(a[0] + 1) % C.VOCAB] + a[1:]
    for name, right, remembers in (("parallel", 0.0, False), ("parallel", 1.0, True), ("latent", 1.0, True)):
        cfg = config_dict(name)
        for entry in cfg["layers"]:
            if entry["type"] == "parallel":
                entry["mixer"]["left"]["mask"]["size"] = 5
                entry["mixer"]["right_scale"] = right
        model = TenalornForCausalLM(TenalornConfig.from_dict(cfg), torch.float32)
        model.load_tensors(random_weights(cfg, 1))
        za, zb = model(torch.tensor([a])), model(torch.tensor([b]))
        assert (float((za[:, 5:] - zb[:, 5:]).abs().max()) > 1e-4) == remembers
        # the second token's pair contains the first
        assert float((za[:, 1] - zb[:, 1]).abs().max()) > 1e-3


# ------------------------------------------------------------------ configuration, weights, registry, programs
def test_configuration_reader():
    cfg = config_dict("mixed")
    c = TenalornConfig.from_dict(cfg)
    assert c.num_hidden_layers == 5 and c.streams == 3 and c.layers[2].mlp is None and c.layers[1].mixer.rank == 36 and c.bigram.buckets == 101
    assert c.layers[0].mixer.left.chunk == 9 and c.layers[0].mixer.left.distance_bias and c.layers[0].mixer.right.gate_cap == 6.0
    assert c.layers[0].mlp == ExpertSpec(5, 2, 20, "softmax", True, True, "output", 2, 24)
    for name in CASES:
        d = config_dict(name)
        c = TenalornConfig.from_dict(d)
        assert TenalornConfig.from_dict(c.to_dict()) == c
        assert c.num_parameters() == sum(t.numel() for t in random_weights(d).values())
    for breakage in (lambda d: d.update(architecture="Other"), lambda d: d["layers"][0].update(type="linear"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                     lambda d: d["layers"][0]["mixer"]["left"].update(heads=5), lambda d: d.update(layers=[]), lambda d: d.update(streams=0),
                     lambda d: d.update(streams=17), lambda d: d["layers"][0]["mixer"]["right"].update(dim=0), lambda d: d.update(logit_softcap=0),
                     lambda d: d["layers"][1]["mixer"]["rot"].update(dims=8), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3),
                     lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(size=0), lambda d: d["layers"][1]["mlp"]["router"].update(top=10),
                     lambda d: d["embedding"]["bigram"].update(buckets=0)):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            TenalornConfig.from_dict(bad)


def test_weights_load_save_and_are_all_checked(tmp_path):
    case = Case("mixed")
    case.save(tmp_path / "m")
    model = registry.load_causal_lm(str(tmp_path / "m"), torch.float32)
    assert isinstance(model, TenalornForCausalLM) and registry.family_of(str(tmp_path / "m")).name == "tenalorn"
    assert all(torch.equal(a, b) for a, b in zip(model.buffers(), case.model.buffers()))
    for name, t in model.checkpoint_tensors().items():
        assert torch.equal(t, case.weights[name].float()), name
    model.save_pretrained(str(tmp_path / "again"))
    back = registry.load_causal_lm(str(tmp_path / "again"), torch.float32)
    assert all(torch.equal(a, b) for a, b in zip(back.buffers(), model.buffers()))
    fresh = TenalornForCausalLM(case.model.config, torch.float32)
    for change in (lambda w: w.pop("l1.mix.uk"), lambda w: w.update({"l2.norm2": w["l1.norm2"]}), lambda w: w.update(bigram=w["bigram"][:-1]),
                   lambda w: w.update({"l0.hc1.mix": w["l0.hc1.mix"][:, 1:]}), lambda w: w.pop("l1.mlp.e7.up"), lambda w: w.pop("l0.mlp.correction"),
                   lambda w: w.update({"l0.mix.right.i": w["l0.mix.right.i"][:1]})):
        bad = dict(case.weights)
        change(bad)
        with pytest.raises((KeyError, ValueError)):
            fresh.load_tensors(bad)


def test_registry_hub_and_tiny_model():
    from ferrotorch_b200 import hub

    assert "tenalorn" in registry.list_causal_lms()
    info = hub.get_model_info("tenalorn-3b")
    assert info.build().num_parameters() == info.num_parameters
    assert TenalornForCausalLM.tiny_random(torch.float32)(torch.tensor([[1, 2, 3]])).shape == (1, 3, 1000)


def test_cache_holds_latents_tokens_and_states_per_slot():
    cache = Case("mixed").model.make_paged_cache(4, 16, 3, 64)
    assert len(cache.k) == 5 and sorted(cache.states) == [0, 2, 4] and not cache.rewindable and cache.token_pages.shape == (4, 16)
    assert cache.states[0].S.shape == (4, 3, 32, 16) and cache.states[0].n.shape == (4, 3, 32) and cache.states[0].m.shape == (4, 3)
    assert cache.k[1].shape == (4, 16, 1, 48 + 16) and cache.v[1].shape == (4, 16, 1, 48) and cache.v[1].data_ptr() == cache.k[1].data_ptr()
    assert Case("latent").model.make_paged_cache(4, 16, 3, 64).rewindable


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
    assert server.main(["--tiny", "--family", "tenalorn", *args]) == 0
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
    assert {"ft_latent_decode", "ft_memory_chunks", "ft_stream_step"} <= need <= have, need - have

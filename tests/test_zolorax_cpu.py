"""The Zolorax decoder on the CPU path: every mechanism and the serving machinery around it against the plain oracle."""
import io
import json
import math

import pytest
import torch

import decoder_cases as C
import zolorax_oracle as O
from zolorax_cases import CASES, Case, config_dict, random_weights
from ferrotorch_b200.models import registry
from ferrotorch_b200.models.generation import GenerationConfig, generate
from ferrotorch_b200.models.serving import ContinuousBatcher
from ferrotorch_b200.models.zolorax import ZoloraxConfig, ZoloraxForCausalLM
from ferrotorch_b200.nn.feed_forward import ExpertSpec, RoutedExperts
from ferrotorch_b200.nn.packed_block import RotarySpec, YarnScaling
from ferrotorch_b200.nn.paged import PagedKVCache, RaggedBatch
from ferrotorch_b200.ops import decoder as D
from ferrotorch_b200.ops import functional as F
from planted_keys import check_planted_keys


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request):
    return Case(request.param)


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


# ------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_rms_norm_of_residual_rows(offset):
    x, w = torch.randn(6, 20, generator=_gen()), torch.randn(20, generator=_gen(1))
    pad = torch.nn.functional.pad
    for eps in (1e-6, 0.5):
        want = O.rms(x.double(), eps) * (offset + w.double())
        got = D.rms_rows(pad(x, (0, 4)), pad(w, (0, 4)), eps, count=20, offset=offset)
        assert torch.allclose(got[:, :20].double(), want, atol=1e-6) and not got[:, 20:].any()
        rows = torch.tensor([5, 0, 5])
        assert torch.equal(D.rms_rows(x, w, eps, offset=offset, rows=rows), D.rms_rows(x, w, eps, offset=offset)[rows])
    assert torch.allclose(O.one_plus_norm(x, w, 1e-6), O.rms(x, 1e-6) * (1 + w))
    # rows that first gain their experts' outputs
    terms, where = torch.randn(12, 20, generator=_gen(2)), torch.randperm(12, generator=_gen(3)).view(6, 2).int()
    total = x + terms[where[:, 0].long()] + terms[where[:, 1].long()]
    want = O.rms(total.double(), 1e-6) * (offset + w.double())
    assert torch.allclose(D.rms_rows(x, w, 1e-6, offset=offset, pending=(terms, where)).double(), want, atol=1e-6)
    y = x.clone()
    D.rms_rows(y, w, 1e-6, offset=offset, pending=(terms, where), update=True)
    assert torch.allclose(y, total, atol=1e-6)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 500.0, 3.0, 40, 4.0, 0.5), (64, 10000.0, 8.0, 4096, 32.0, 1.0), (2, 20.0, 2.0, 100, 8.0, 1.0),
                                                                (8, 100.0, 1.0, 64, 2.0, 1.0), (32, 1e6, 0.5, 8, 1.0, 1.0), (12, 50.0, 4.0, 5, 32.0, 1.0)])
def test_rotation_table_follows_the_scaling(dims, base, factor, original, fast, slow):
    rot = {"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    freq, amplitude = O.rotary_frequencies(rot)
    table = RotarySpec(dims, base, YarnScaling(factor, original, fast, slow)).table(5000).double()
    for p in (0, 1, 17, 4999):
        assert torch.allclose(table[p, :, 0], amplitude * torch.cos(p * freq), atol=1e-7)
        assert torch.allclose(table[p, :, 1], amplitude * torch.sin(p * freq), atol=1e-7)
    plain = RotarySpec(dims, base).table(10).double()
    f0, one = O.rotary_frequencies({"dims": dims, "base": base})
    assert one == 1.0 and torch.allclose(plain[9, :, 0], torch.cos(9 * f0), atol=1e-7)


def test_scaling_moves_slow_dimensions_only():
    f, amp = O.rotary_frequencies({"dims": 64, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    plain, _ = O.rotary_frequencies({"dims": 64, "base": 10000.0})
    assert f[0] == plain[0] and f[-1] == pytest.approx(float(plain[-1]) / 4.0) and amp == pytest.approx(0.1 * math.log(4.0) + 1.0)


@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 24, 16, 8), (3, 1, 16, 32, 16), (2, 2, 32, 16, None)])
def test_norm_and_rotation_of_heads_and_the_cached_keys(heads, kv, dim, vdim, rot):
    g, T, eps = _gen(5), 11, 1e-3
    Dp, Vp = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    cache = PagedKVCache(1, kv, Dp, 4, 2, 64, 8, "cpu", torch.float32, v_head_dim=Vp)
    cache.reserve(1, 20)
    batch = RaggedBatch([(1, [0] * T, 9, [])], "cpu")
    wq, wk = torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    spec = {"dims": rot, "base": 30.0} if rot else None
    table = RotarySpec(rot, 30.0).table(64) if rot else None
    q, k, v = (torch.randn(T, n, d, generator=g) for n, d in ((heads, dim), (kv, dim), (kv, vdim)))
    pad = torch.nn.functional.pad
    packed = torch.cat([pad(q, (0, Dp - dim)).flatten(1), pad(k, (0, Dp - dim)).flatten(1), pad(v, (0, Vp - vdim)).flatten(1)], 1)
    D.qkv_head_finish(packed, cache, 0, batch, heads=heads, dim=Dp, k_off=heads * Dp, v_off=(heads + kv) * Dp,
                      q_weight=pad(wq, (0, Dp - dim)), k_weight=pad(wk, (0, Dp - dim)), true_dim=dim, eps=eps, table=table)
    ks, vs = cache.gather(0, 1, 20)

    def want(t, w, p):
        z = O.rms(t.double(), eps) * w.double()
        return O.rotate(z, p, spec) if spec else z

    for t in range(T):
        for a in range(heads):
            assert torch.allclose(packed[t, a * Dp:a * Dp + dim].double(), want(q[t, a], wq, 9 + t), atol=1e-5)
        for c in range(kv):
            assert torch.allclose(ks[9 + t, c, :dim].double(), want(k[t, c], wk, 9 + t), atol=1e-5)
            assert torch.equal(vs[9 + t, c, :vdim], v[t, c])
    assert not ks[:9].any() and not ks[9:, :, dim:].any()


@pytest.mark.parametrize("window,sink,elem", [(1, True, True), (7, False, True), (16, True, False), (23, True, True), (500, True, True), (None, True, True)])
def test_attention_sees_its_window_and_its_sink(window, sink, elem):
    check_planted_keys(6, 2, 32, 16, 8, torch.float32, "cpu", length=70, window=window, sink=sink, elem_gate=elem)


def test_window_edges_exactly():
    assert O.visible_keys(10, 4) == (7, 11) and O.visible_keys(2, 4) == (0, 3) and O.visible_keys(9, 1) == (9, 10)


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_carries_its_inputs_across_portions(taps):
    g, C_, T = _gen(taps), 8, 40
    x, w, b = torch.randn(T, C_, generator=g), torch.randn(taps, C_, generator=g), torch.randn(C_, generator=g)
    want = O.causal_convolution(x.double(), w.t().double(), b.double())
    state = torch.full((3, taps - 1, C_), 9.0)            # what an earlier sequence left in the slot
    at, rows = 0, []
    for n in (1, 1, 2, 3, 1, 9, 1, 22):
        batch = RaggedBatch([(2, [0] * n, at, [])], "cpu")
        rows.append(D.causal_conv(x[at:at + n], w, b, state, batch))
        if n > 1 and taps > 1:                            # portions leave their inputs in the scan
            keep = torch.cat([state[2], x[at:at + n]])[n:n + taps - 1]
            state[2] = keep
        at += n
    assert torch.allclose(torch.cat(rows).double(), want, atol=1e-5)


def test_recurrence_over_portions_equals_the_oracle():
    g, blocks, n, T = _gen(8), 3, 8, 50
    W = blocks * n
    u, y = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g)
    gates, rb, ib = torch.randn(blocks, 2, n, n, generator=g) * 0.4, torch.randn(W, generator=g), torch.randn(W, generator=g)
    lam = torch.linspace(-9.0, 2.0, W)
    decay = -8.0 * torch.nn.functional.softplus(lam)
    ud = u.double()
    r = torch.sigmoid(O.block_linear(ud, gates[:, 0].double(), rb.double().view(blocks, n)))
    i = torch.sigmoid(O.block_linear(ud, gates[:, 1].double(), ib.double().view(blocks, n)))
    want = O.gated_linear_recurrence(ud, r, i, lam.double()) * O.gelu_tanh(y.double())
    state, at, rows = torch.full((2, W), 5.0), 0, []
    for k in (1, 2, 1, 17, 1, 1, 27):
        batch = RaggedBatch([(0, [0] * k, at, [])], "cpu")
        out = torch.empty(k, W)
        D.gated_recurrence(u[at:at + k], y[at:at + k], gates, rb, ib, decay, state, batch, u[at:at + k], torch.zeros(2, 0, W), out)
        rows.append(out)
        at += k
    assert torch.allclose(torch.cat(rows).double(), want, atol=2e-5)
    assert torch.equal(state[1], torch.full((W,), 5.0))   # another sequence's slot


@pytest.mark.parametrize("experts,top", [(5, 1), (5, 2), (3, 3), (40, 7)])
def test_routed_experts(experts, top):
    g, W, ff, T = _gen(experts), 20, 12, 30
    module = RoutedExperts(W, ExpertSpec(experts, top, ff))
    sd = {n: torch.randn(s, generator=g) * s[1] ** -0.5 * 2 for n, s in module._shapes().items()}
    module.load(sd)
    h = torch.randn(T, W, generator=g)
    got = module(torch.nn.functional.pad(h, (0, 4))).total()
    want = O.mixture(h.double(), {k: v.double() for k, v in sd.items()}, {"top": top})
    assert torch.allclose(got[:, :W].double(), want, atol=1e-5) and not got[:, W:].any()
    assert all(torch.equal(v, sd[k]) for k, v in module.unpack().items())


def test_routing_weight_scales_the_input_and_is_not_normalised():
    z = torch.tensor([[0.3, -1.0]])
    W = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0]]), "e0.gate": torch.ones(1, 2), "e0.up": torch.ones(1, 2), "e0.down": torch.ones(2, 1),
         "e1.gate": torch.zeros(1, 2), "e1.up": torch.zeros(1, 2), "e1.down": torch.zeros(2, 1)}
    s = 1 / (1 + math.exp(-0.3))
    inner = s * (0.3 - 1.0)
    want = inner / (1 + math.exp(-inner)) * inner
    assert O.mixture(z.double(), {k: v.double() for k, v in W.items()}, {"top": 1})[0, 0].item() == pytest.approx(want)
    module = RoutedExperts(2, ExpertSpec(2, 1, 1))
    module.load(W)
    assert module(torch.nn.functional.pad(z, (0, 6))).total()[0, 0].item() == pytest.approx(want, rel=1e-5)


def test_equal_logits_take_the_lower_expert():
    route = D.moe_route(torch.tensor([[1.0, 0.0]]), torch.tensor([[2.0, 0], [3.0, 0], [3.0, 0], [3.0, 0]]), 4, 2)
    assert route.index.tolist() == [[1, 2]]


def test_squared_relu():
    h, up, down = torch.randn(5, 8, generator=_gen(1)), torch.randn(16, 8, generator=_gen(2)), torch.randn(8, 16, generator=_gen(3))
    want = O.squared_relu_mlp(h.double(), {"up": up.double(), "down": down.double()})
    assert torch.allclose((F.linear_rows(h, up, activation="relu2") @ down.t()).double(), want, atol=1e-4)


# ------------------------------------------------------------------ the model on the step function
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
        assert torch.allclose(seen[i][:, :width].double(), w, atol=4e-5) and not seen[i][:, width:].any()


def test_greedy_generation_through_the_scheduler(case):
    C.check_generation(case)


def test_generation_with_preemption():
    case = Case("mixed")
    b = C.check_generation(case, blocks=5)                # starved: sequences give way and are recomputed
    assert b.stats.preemptions > 0


def test_states_are_not_shared_or_wound_back():
    case = Case("mixed")
    system = case.tokens(26, 40)
    prompts = [system + case.tokens(n, 50 + n) for n in (3, 9, 1)]
    plain = ContinuousBatcher(case.model, 64, 8, 3, 64).generate(prompts, 6)
    shared = ContinuousBatcher(case.model, 64, 8, 1, 64, prefix_caching=True)
    assert shared.prefix is None and shared.generate(prompts, 6) == plain
    looked = ContinuousBatcher(case.model, 64, 8, 3, 64)
    reqs = [looked.submit(p, 6, lookahead=4) for p in prompts]
    looked.run()
    assert [r.output for r in reqs] == plain and looked.stats.spec_proposed == 0
    with pytest.raises(ValueError):
        looked.cache.adopt(0, [0], 8)
    # a model without recurrent layers keeps both
    case = Case("attention")
    prompts = [case.tokens(26, 40) + case.tokens(n, 50 + n) for n in (3, 9, 1)]
    plain = ContinuousBatcher(case.model, 64, 8, 3, 64).generate(prompts, 6)
    shared = ContinuousBatcher(case.model, 64, 8, 1, 64, prefix_caching=True)
    assert shared.generate(prompts, 6) == plain and shared.stats.prefix_hit_tokens >= 2 * 24


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
    # windows hide a changed first token from attention; the recurrence remembers it
    for name, remembers in (("attention", False), ("recurrent", True)):
        case = Case(name)
        if name == "attention":
            for entry in case.cfg["layers"]:
                entry["mixer"]["mask"]["size"] = 5
            case.model.load_tensors(case.weights)
            model = ZoloraxForCausalLM(ZoloraxConfig.from_dict(case.cfg), torch.float32)
            model.load_tensors(case.weights)
        else:
            model = case.model
        a = case.tokens(40, 3)
        b = [(a[0] + 1) % C.VOCAB] + a[1:]
        za, zb = model(torch.tensor([a])), model(torch.tensor([b]))
        reach = 1 + 4 * 4                                 # four layers of four tokens back
        same = float((za[:, reach:] - zb[:, reach:]).abs().max())
        assert (same > 1e-4) == remembers


# ------------------------------------------------------------------ configuration, weights, registry, programs
def test_configuration_reader():
    cfg = config_dict("mixed")
    c = ZoloraxConfig.from_dict(cfg)
    assert c.num_hidden_layers == 5 and c.layers[2].mlp is None and c.layers[1].mixer.vdim == 40 and c.layers[2].mixer.kv_from == 1
    assert c.layers[1].mixer.rotary.scaling.original == 60 and c.layers[3].mlp == ExpertSpec(8, 1, 33)
    for name in CASES:
        d = config_dict(name)
        c = ZoloraxConfig.from_dict(d)
        assert ZoloraxConfig.from_dict(c.to_dict()) == c
        assert c.num_parameters() == sum(t.numel() for t in random_weights(d).values())
    for breakage in (lambda d: d.update(architecture="Other"), lambda d: d["layers"][0].update(type="linear"), lambda d: d["layers"][0]["mlp"].update(kind="none"),
                     lambda d: d["layers"][1]["mixer"].update(heads=5), lambda d: d.update(layers=[]), lambda d: d["layers"][0]["mixer"].update(blocks=5),
                     lambda d: d["layers"][2]["mixer"].update(kv_from=0), lambda d: d["layers"][2]["mixer"].update(kv_from=2),
                     lambda d: d["layers"][2]["mixer"].update(kv_from=4), lambda d: d["layers"][2]["mixer"].update(vdim=32),
                     lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26),
                     lambda d: d["layers"][1]["mlp"]["router"].update(top=6)):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            ZoloraxConfig.from_dict(bad)
    open_ = json.loads(json.dumps(cfg))
    del open_["layers"][4]["mixer"]["mask"], open_["layers"][4]["mixer"]["rot"]["scaling"]
    m = ZoloraxConfig.from_dict(open_).layers[4].mixer
    assert m.window is None and m.rotary.scaling is None


def test_weights_load_save_and_are_all_checked(tmp_path):
    case = Case("mixed")
    case.save(tmp_path / "m")
    model = registry.load_causal_lm(str(tmp_path / "m"), torch.float32)
    assert isinstance(model, ZoloraxForCausalLM) and registry.family_of(str(tmp_path / "m")).name == "zolorax"
    assert all(torch.equal(a, b) for a, b in zip(model.buffers(), case.model.buffers()))
    for name, t in model.checkpoint_tensors().items():
        assert torch.equal(t, case.weights[name].float()), name
    model.save_pretrained(str(tmp_path / "again"))
    back = registry.load_causal_lm(str(tmp_path / "again"), torch.float32)
    assert all(torch.equal(a, b) for a, b in zip(back.buffers(), model.buffers()))
    fresh = ZoloraxForCausalLM(case.model.config, torch.float32)
    for change in (lambda w: w.pop("l1.mix.sink"), lambda w: w.update({"l2.mix.k": w["l1.mix.k"]}), lambda w: w.update(embed=w["embed"][:-1]),
                   lambda w: w.update({"l0.mix.conv": w["l0.mix.conv"][:, 1:]}), lambda w: w.pop("l3.mlp.e7.up"), lambda w: w.update({"l0.mix.lam": w["l0.mix.lam"][:1]})):
        bad = dict(case.weights)
        change(bad)
        with pytest.raises((KeyError, ValueError)):
            fresh.load_tensors(bad)


def test_registry_hub_and_tiny_model():
    from ferrotorch_b200 import hub

    assert "zolorax" in registry.list_causal_lms()
    info = hub.get_model_info("zolorax-3b")
    assert info.build().num_parameters() == info.num_parameters
    assert ZoloraxForCausalLM.tiny_random(torch.float32)(torch.tensor([[1, 2, 3]])).shape == (1, 3, 1000)


def test_cache_holds_keys_once_and_states_per_slot():
    case = Case("mixed")
    cache = case.model.make_paged_cache(4, 16, 3, 64)
    assert len(cache.k) == 2 and sorted(cache.states) == [0, 3] and not cache.rewindable
    assert cache.states[0].state.shape == (4, 48) and cache.states[0].conv.shape == (4, 3, 48) and cache.states[3].conv.shape[1] == 0
    none = Case("recurrent").model.make_paged_cache(4, 16, 3, 64)
    assert none.k == [] and len(none.states) == 3


def test_trace_replay_writes_logits_and_reuses_slots(tmp_path, monkeypatch, capsys):
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
    code = trace.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "128", "--device", "cpu"])
    assert code == 0
    assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(5)]
    want = {0: [(a, 0), (a, 16)], 2: [(b, 20), (b, 5), (a, 39)], 3: [(b, 20)], 4: [(a, 39)]}
    assert sorted(int(p.stem) for p in (tmp_path / "out").iterdir()) == sorted(want)
    for step, rows in want.items():
        data = (tmp_path / "out" / ("%d.f32" % step)).read_bytes()
        got = torch.frombuffer(bytearray(data), dtype=torch.float32).view(len(rows), C.VOCAB)
        case.check(got, torch.stack([case.oracle(t)[i] for t, i in rows]), "step %d" % step)


def test_server_command_line_serves_the_family(tmp_path):
    from ferrotorch_b200.models import server

    args = ["--device", "cpu", "--port", "0", "--kv-pages", "16", "--serve-seconds", "0.2"]
    assert server.main(["--tiny", "--family", "zolorax", *args]) == 0
    Case("mixed").save(tmp_path / "m")
    assert server.main(["--model", str(tmp_path / "m"), *args]) == 0


def test_the_decoder_kernel_set_holds_every_kernel_the_path_calls():
    import os
    import re

    from ferrotorch_b200 import _native

    text = "".join(open(os.path.join(_native.CSRC, n + ".cu")).read() for n in _native.KERNEL_SETS["decoder"])
    have = set(re.findall(r"FT_API[^;{(]*?\b(ft_\w+)\s*\(", text))
    source = open(os.path.join(os.path.dirname(D.__file__), "decoder.py")).read()
    need = set(re.findall(r"\.(ft_\w+)\(", source)) | {"ft_gemm_bf16", "ft_gemm_small_m_f32", "ft_paged_decode", "ft_paged_prefill", "ft_paged_rows"}
    assert need <= have, need - have

"""The Bopudra decoder on the CPU path: every mechanism and the serving machinery around it against the plain oracle."""
import io
import json
import math

import pytest
import torch

import bopudra_cases as C
import bopudra_oracle as O
from ferrotorch_b200.models import registry
from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM
from ferrotorch_b200.models.generation import GenerationConfig, generate
from ferrotorch_b200.models.serving import ContinuousBatcher
from planted_keys import check_planted_keys
from ferrotorch_b200.nn.paged import RaggedBatch
from ferrotorch_b200.ops import functional as F
from ferrotorch_b200.ops import reference as R


@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    return C.Case(request.param)


# ------------------------------------------------------------------ mechanisms
def test_dynamic_tanh_and_its_fused_gather():
    g = torch.Generator().manual_seed(0)
    table, w, b = torch.randn(9, 16, generator=g), torch.randn(16, generator=g), torch.randn(16, generator=g)
    alpha = torch.tensor(0.7)
    ids = torch.tensor([3, 0, 8, 3])
    want = O.dynamic_tanh(table[ids].double(), 0.7, w.double(), b.double())
    x, h = F.embedding_dynamic_tanh(ids, table, alpha, w, b)
    assert torch.equal(x, table[ids]) and torch.allclose(h.double(), want, atol=1e-6)
    assert torch.allclose(F.dynamic_tanh(x, alpha, w, b, scale=2.5).double(), 2.5 * want, atol=1e-6)


def test_projection_norm_counts_true_elements_only():
    z = torch.randn(5, 20, generator=torch.Generator().manual_seed(1))
    w = torch.linspace(0.5, 2.0, 20)
    pad = torch.nn.functional.pad
    for eps in (1e-6, 0.5):
        got = R.projection_rms(pad(z, (0, 12)), pad(w, (0, 12)), eps, 20)
        assert torch.allclose(got[:, :20].double(), O.rms_over_all(z.double(), w.double(), eps), atol=1e-6)
        assert not got[:, 20:].any()


@pytest.mark.parametrize("coef,every", [(0.5, 4), (0.1, 8192), (2.0, 1), (0.3, 2.5)])
def test_query_temperature_steps_at_multiples(coef, every):
    pos = torch.tensor([0, 1, 2, 3, 4, 6, 7, 8, 8190, 8191, 8192, 16382, 16383, 100000, 8191 * 37])
    got = R.query_temperature(pos, coef, every)
    assert got.tolist() == pytest.approx([O.query_temperature(int(p), coef, every) for p in pos], rel=1e-6)
    assert R.query_temperature(torch.tensor([8190]), 1.0, 8192).item() == 1.0
    assert R.query_temperature(torch.tensor([8191]), 1.0, 8192).item() == pytest.approx(1 + math.log(2.0))


def test_head_gate_and_activation():
    o, z = torch.randn(3, 4, 5), torch.randn(3, 4)
    assert torch.allclose(R.head_gate(o, z), o * torch.sigmoid(z)[:, :, None])
    u = torch.linspace(-6, 6, 50)
    assert torch.allclose(R._ACTS[F._ACT_ID["gelu"]](u).double(), O.gelu_tanh(u.double()), atol=1e-6)


@pytest.mark.parametrize("Hq,Hkv,D,Dv,block", [(6, 2, 16, 48, 8), (3, 3, 32, 16, 16), (5, 1, 48, 80, 4)])
def test_attention_over_pages_sees_the_key_it_should(Hq, Hkv, D, Dv, block):
    check_planted_keys(Hq, Hkv, D, Dv, block, torch.float32, "cpu", length=70)


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
        assert torch.allclose(seen[i][:, :width].double(), w, atol=2e-5) and not seen[i][:, width:].any()


def test_greedy_generation_through_the_scheduler(case):
    C.check_generation(case)


def test_generation_with_preemption_and_prefix_pages():
    case = C.Case("even")
    b = C.check_generation(case, blocks=5)                # starved: sequences give way and are recomputed
    assert b.stats.preemptions > 0
    system = case.tokens(26, 40)
    prompts = [system + case.tokens(n, 50 + n) for n in (3, 9, 1)]
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
    case = C.Case("one head")
    toks = case.tokens(300, 70)
    got = C.feed_all(case, [3, 1], toks)
    case.check(got, case.oracle(toks), "long decoding")


# ------------------------------------------------------------------ configuration, weights, registry, programs
def test_configuration_reader(tmp_path):
    cfg = C.config_dict("uneven")
    c = BopudraConfig.from_dict(cfg)
    assert c.num_hidden_layers == 4 and c.layers[1].ff is None and c.layers[0].attention.vdim == 40 and c.logit_scale == 3.0
    again = BopudraConfig.from_dict(c.to_dict())
    assert again == c
    assert c.num_parameters() == sum(t.numel() for t in C.random_weights(cfg).values())
    for breakage in (lambda d: d.update(architecture="Other"), lambda d: d["layers"][0].update(type="recurrent"),
                     lambda d: d["layers"][0]["mlp"].update(kind="routed"), lambda d: d["layers"][0]["mixer"].update(heads=5),
                     lambda d: d.update(layers=[]), lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=0)):
        bad = json.loads(json.dumps(cfg))
        breakage(bad)
        with pytest.raises(ValueError):
            BopudraConfig.from_dict(bad)
    del cfg["layers"][2]["mixer"]["q_temp"]
    assert BopudraConfig.from_dict(cfg).layers[2].attention.temp_coef == 0.0


def test_weights_load_save_and_are_all_checked(tmp_path):
    case = C.Case("uneven")
    case.save(tmp_path / "m")
    model = registry.load_causal_lm(str(tmp_path / "m"), torch.float32)
    assert isinstance(model, BopudraForCausalLM) and registry.family_of(str(tmp_path / "m")).name == "bopudra"
    assert all(torch.equal(a, b) for a, b in zip(model.buffers(), case.model.buffers()))
    for name, t in model.checkpoint_tensors().items():
        assert torch.equal(t, case.weights[name].float()), name
    model.save_pretrained(str(tmp_path / "again"))
    back = registry.load_causal_lm(str(tmp_path / "again"), torch.float32)
    assert all(torch.equal(a, b) for a, b in zip(back.buffers(), model.buffers()))
    fresh = BopudraForCausalLM(case.model.config, torch.float32)
    for change in (lambda w: w.pop("l1.mix.g"), lambda w: w.update({"l1.mlp.up": w["l0.mlp.up"]}), lambda w: w.update(embed=w["embed"][:-1]),
                   lambda w: w.update({"l0.mix.v": w["l0.mix.v"][:-1]})):
        bad = dict(case.weights)
        change(bad)
        with pytest.raises((KeyError, ValueError)):
            fresh.load_tensors(bad)


def test_registry_knows_the_families():
    assert {"llama", "bopudra"} <= set(registry.list_causal_lms())
    assert registry.family_of({"model_type": "llama"}).name == "llama"
    assert registry.family_of({"hidden_size": 8, "num_attention_heads": 2}).name == "llama"
    with pytest.raises(ValueError):
        registry.family_of({"architecture": "unheard of"})
    with pytest.raises(ValueError):
        registry.family_named("unheard of")


def test_hub_entry_states_the_size():
    from ferrotorch_b200 import hub

    info = hub.get_model_info("bopudra-8b")
    assert info.build().num_parameters() == info.num_parameters


def test_trace_replay_writes_logits_and_reuses_slots(tmp_path, monkeypatch, capsys):
    from ferrotorch_b200.models import trace

    case = C.Case("uneven")
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
    assert server.main(["--tiny", "--family", "bopudra", *args]) == 0
    C.Case("even").save(tmp_path / "m")
    assert server.main(["--model", str(tmp_path / "m"), *args]) == 0


def test_the_decoder_kernel_set_holds_every_kernel_the_path_calls():
    import os
    import re

    from ferrotorch_b200 import _native

    text = "".join(open(os.path.join(_native.CSRC, n + ".cu")).read() for n in _native.KERNEL_SETS["decoder"])
    have = set(re.findall(r"FT_API[^;{(]*?\b(ft_\w+)\s*\(", text))
    need = {"ft_dyt_fwd", "ft_qkv_finish", "ft_gemm_bf16", "ft_gemm_small_m", "ft_gemm_small_m_f32", "ft_paged_decode", "ft_paged_prefill", "ft_paged_rows",
            "ft_kv_append", "ft_rmsnorm_fwd", "ft_rope", "ft_swiglu_fwd", "ft_embedding_fwd", "ft_launch_count", "ft_read_device_status"}
    assert need <= have, need - have

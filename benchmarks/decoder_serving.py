"""Prefill and decode throughput of the decoder families that the serving engine runs, side by side at equal size.

    python bench.py --workload decoder-serving                 # all families and sizes below
    python bench.py --workload decoder-serving --serving-sizes 8b --serving-kernels

Random weights.  All families run on ``models.serving.PagedStepper``: prefill feeds prompts of ``prompt`` tokens in steps
of at most 8192 tokens, decode replays the captured single-token step of ``batch`` sequences at contexts around
``prompt``.  Times are CUDA events around whole steps after warm-up (weights and cache exceed L2 at these sizes);
``--serving-kernels`` times every kernel of one layer with a 512 MB write between launches and relates it to the
measured copy bandwidth or cuBLAS bf16 rate of the box."""
from __future__ import annotations

import gc
import json
import os
import statistics

import torch

# name: (hidden, layers, heads, kv heads, head size, SwiGLU width, vocabulary, prompt, batch).  The parallel family's
# two-matrix MLP is 1.5 x as wide, so both have the same number of parameters and matrix-product FLOPs.  Zolorax has the
# same dense MLP in every other layer and eight experts of half the SwiGLU width, two of them used, in the others: equal
# FLOPs per token, but more weights to read in a decode step.  Tenalorn has in every layer eight experts of a third of the
# SwiGLU width, two of them used, and a shared one: again equal FLOPs; memories of 128 x 128 with half the width in all.  Mogelix
# has the dense MLP in every sixth layer, in the others eight two-matrix experts of half the SwiGLU width, two of them used, and a
# shared one: equal FLOPs; state-space heads of 64 with twice the width in all and states of 128, and a gate of the width of the
# model for every sublayer.
SIZES = {"1b": (2048, 16, 32, 8, 64, 8192, 128256, 2048, 64),
         "3b": (3072, 28, 24, 8, 128, 8192, 128256, 2048, 64),
         "8b": (4096, 32, 32, 8, 128, 14336, 128256, 2048, 64)}
FAMILIES = ("llama", "bopudra", "zolorax", "tenalorn", "mogelix")
PAGE = 16
EXPERTS, TOP, WINDOW, POOL = 8, 2, 1024, 16


def zolorax_config(size: str, n: int):
    from ferrotorch_b200.models.zolorax import ZoloraxConfig, ZoloraxLayerConfig
    from ferrotorch_b200.nn.feed_forward import ExpertSpec

    hidden, _, heads, kv, dim, ff, vocab, _, _ = SIZES[size]
    cfg = ZoloraxConfig.pattern(vocab, hidden, n, heads, kv, dim, ff, experts=0, window=WINDOW)
    cfg.layers = [ZoloraxLayerConfig(s.mixer, ExpertSpec(EXPERTS, TOP, ff // TOP) if i % 2 else ff * 3 // 2) for i, s in enumerate(cfg.layers)]
    return cfg


def tenalorn_config(size: str, n: int):
    from ferrotorch_b200.models.tenalorn import BigramSpec, TenalornConfig

    hidden, _, heads, kv, dim, ff, vocab, _, _ = SIZES[size]
    return TenalornConfig.pattern(vocab, hidden, n, heads, kv, dim, ff // 3 // 64 * 64, chunk=WINDOW, memory_heads=hidden // 256, memory_dim=128,
                                  memory_vdim=128, rank=512, experts=EXPERTS, top=TOP, identity=0, streams=2, bigram=BigramSpec(131071, 1031, 17))


def mogelix_config(size: str, n: int):
    from ferrotorch_b200.models.mogelix import MogelixConfig

    hidden, _, heads, kv, dim, ff, vocab, _, _ = SIZES[size]
    return MogelixConfig.pattern(vocab, hidden, n, heads, kv, dim, ff * 3 // 2, window=WINDOW, pool=POOL, state_dim=64, state=128, experts=EXPERTS, top=TOP,
                                 expert_ff=ff // 2, shared_ff=ff // 2, alpha=3.0)


def build(family: str, size: str, layers: int | None = None):
    hidden, n, heads, kv, dim, ff, vocab, _, _ = SIZES[size]
    n = layers or n
    if family == "bopudra":
        from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM

        return BopudraForCausalLM(BopudraConfig.uniform(vocab, hidden, n, heads, kv, dim, ff * 3 // 2), device="cuda").random_()
    if family == "zolorax":
        from ferrotorch_b200.models.zolorax import ZoloraxForCausalLM

        return ZoloraxForCausalLM(zolorax_config(size, n), device="cuda").random_()
    if family == "tenalorn":
        from ferrotorch_b200.models.tenalorn import TenalornForCausalLM

        return TenalornForCausalLM(tenalorn_config(size, n), device="cuda").random_()
    if family == "mogelix":
        from ferrotorch_b200.models.mogelix import MogelixForCausalLM

        return MogelixForCausalLM(mogelix_config(size, n), device="cuda").random_()
    from ferrotorch_b200.models.llama import LlamaConfig, LlamaForCausalLM

    cfg = LlamaConfig(vocab_size=vocab, hidden_size=hidden, intermediate_size=ff, num_hidden_layers=n, num_attention_heads=heads,
                      num_key_value_heads=kv, head_dim=dim, max_position_embeddings=8192)
    prev = torch.get_default_dtype()
    torch.set_default_dtype(torch.bfloat16)
    try:
        with torch.device("cuda"):
            return LlamaForCausalLM(cfg).eval()
    finally:
        torch.set_default_dtype(prev)


def _event_ms(fn, warm: int, k: int) -> float:
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(k):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / k


def throughput(model, size: str, steps: int, warmup: int) -> dict:
    """Tokens per second of prefill and of graph-replayed decode, device time of whole steps."""
    from ferrotorch_b200.models.serving import PagedStepper
    from ferrotorch_b200.nn.paged import RaggedBatch

    vocab, prompt, batch = SIZES[size][6:]
    cap = prompt + 16 + 4 * (steps + warmup)
    st = PagedStepper(model, batch * ((cap + PAGE - 1) // PAGE), PAGE, batch, cap, cuda_graph=True)
    g = torch.Generator().manual_seed(0)
    prompts = torch.randint(0, vocab, (batch, prompt), generator=g).tolist()
    slots = [st.admit() for _ in range(batch)]
    per = max(1, 8192 // prompt)
    for i in range(0, batch, per):                        # fills the cache
        st.feed([(s, p, [prompt - 1]) for s, p in zip(slots[i:i + per], prompts[i:i + per])])
    chunk = RaggedBatch([(s, p, 0, [prompt - 1]) for s, p in zip(slots[:per], prompts[:per])], "cuda")
    pre_ms = _event_ms(lambda: model.paged_forward(chunk, st.cache), warmup, steps)

    def decode():
        st.feed([(s, [p[0]], [0]) for s, p in zip(slots, prompts)])

    dec_host_ms = _event_ms(decode, warmup, steps)         # as served: bookkeeping, one upload, replay
    graph = next(iter(st._graphs.values()))[1]
    dec_ms = _event_ms(graph.replay, warmup, steps)
    weights = sum(t.numel() for t in {t.data_ptr(): t for t in [*model.parameters(), *model.buffers()]}.values())
    return {"parameters_billions": round(weights / 1e9, 2), "prefill_tok_s": round(per * prompt / pre_ms * 1e3), "prefill_ms": round(pre_ms, 3), "prefill_tokens_per_step": per * prompt,
            "decode_tok_s": round(batch / dec_ms * 1e3), "decode_ms": round(dec_ms, 3), "decode_step_as_served_ms": round(dec_host_ms, 3),
            "decode_batch": batch, "context": prompt}


def kernel_table(size: str, peaks: dict, steps: int, families=FAMILIES) -> list:
    """Device time and roofline fraction of the kernels of one layer of each family: ``(family, phase, kernel, us, bound, frac)``."""
    from ferrotorch_b200 import _native
    from ferrotorch_b200.nn.paged import RaggedBatch
    from ferrotorch_b200.ops import functional as F

    hidden, _, heads, kv, dim, ff, vocab, prompt, batch = SIZES[size]
    flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
    bw, tf = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12

    def time_us(fn) -> float:
        for _ in range(3):
            fn()
        out = []
        for _ in range(max(5, steps)):
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            out.append(e0.elapsed_time(e1) * 1e3)
        return statistics.median(out)

    rows = []

    def add(family, phase, name, fn, flops, nbytes):
        us = time_us(fn)
        t_f, t_b = flops / tf * 1e6, nbytes / bw * 1e6
        rows.append({"family": family, "phase": phase, "kernel": name, "us": round(us, 1), "bound": "tensor" if t_f > t_b else "hbm",
                     "of_measured": round(max(t_f, t_b) / us, 3)})

    lib = _native.kernels()
    for family in families:
        model = build(family, size, layers={"zolorax": 6, "tenalorn": 3, "mogelix": 6}.get(family, 2))
        cache = model.make_paged_cache(batch * ((prompt + 16) // PAGE + 1), PAGE, batch, prompt + 16)
        for s in range(batch):
            cache.reserve(s, prompt + 1)
        cache.sync_table()
        per = max(1, 8192 // prompt)
        ids = torch.randint(0, vocab, (max(per, batch), prompt), generator=torch.Generator().manual_seed(0)).tolist()
        pre = RaggedBatch([(s, ids[s], 0, [prompt - 1]) for s in range(per)], "cuda")
        dec = RaggedBatch([(s, ids[s][:1], prompt - 1, [0]) for s in range(batch)], "cuda")
        for phase, b in (("prefill", pre), ("decode", dec)):
            T = b.n_rows
            kvb = batch * prompt * kv * 2 * dim * 2
            att_flops = 4 * heads * dim * per * prompt * (prompt + 1) // 2 if phase == "prefill" else 0
            att_bytes = 4 * T * (heads + kv) * dim if phase == "prefill" else kvb

            def gemm(name, a, w, fn):
                add(family, phase, name, fn, 2 * T * w.shape[0] * w.shape[1], 2 * (w.numel() + a.numel()))

            if family == "zolorax":
                _zolorax_kernels(lambda *a: add(family, phase, *a), gemm, model, cache, b, phase == "prefill", (hidden, heads, kv, dim, prompt, per, batch))
            elif family == "tenalorn":
                _tenalorn_kernels(lambda *a: add(family, phase, *a), gemm, model, cache, b, phase == "prefill", (hidden, heads, kv, dim, prompt, per, batch))
            elif family == "mogelix":
                _mogelix_kernels(lambda *a: add(family, phase, *a), gemm, model, cache, b, phase == "prefill", (hidden, heads, kv, dim, prompt, per, batch))
            elif family == "bopudra":
                blk, nrm = model.blocks[0], model.norms[0]
                x, h = F.embedding_dynamic_tanh(b.tokens, model.embed, nrm.alpha, nrm.weight, nrm.bias, out_dtype=torch.bfloat16)
                packed = F.linear_rows(h, blk.in_proj)
                acts = torch.randn(T, blk.out_proj.shape[1], device="cuda").bfloat16()
                sq, sk, sv, su, sg = blk.segments
                a = blk.attn
                add(family, phase, "embedding + norm", lambda: F.embedding_dynamic_tanh(b.tokens, model.embed, nrm.alpha, nrm.weight, nrm.bias),
                    0, T * hidden * 8)
                gemm("in_proj (q|k|v|up|gate)", h, blk.in_proj, lambda: F.linear_rows(h, blk.in_proj))
                add(family, phase, "qkv_finish (norms, append, gelu)", lambda: F.qkv_finish(
                    packed, cache, 0, b, q=sq, k=sk, v=sv, up=su, q_weight=blk.q_norm, k_weight=blk.k_norm, q_count=sq[1], k_count=sk[1],
                    eps=1e-5, temp_coef=a.temp_coef, temp_every=a.temp_every, act_out=acts[:, blk.value_width:]),
                    0, 4 * T * (sq[1] + sk[1] + sv[1] + su[1]))
                q = packed[:, :sq[1]].unflatten(1, (heads, -1))
                gate = packed[:, sg[0]:sg[0] + heads]
                out = acts[:, :blk.value_width].unflatten(1, (heads, -1))
                add(family, phase, "attention (gated)", lambda: cache.attend(0, q, b, a.scale, gate=gate, out=out), att_flops, att_bytes)
                gemm("out_proj (o|down) + residual" + (" + norm" if phase == "decode" else ""), acts, blk.out_proj,
                     lambda: F.residual_linear_(x, acts, blk.out_proj, nrm.as_epilogue() if phase == "decode" else None))
                if phase == "prefill":
                    add(family, phase, "dynamic tanh", lambda: nrm(x, out_dtype=torch.bfloat16), 0, T * hidden * 6)
                else:
                    gemm("head", h, model.head, lambda: F.linear_f32_out(h, model.head))
            else:
                lay, m = model.model.layers[0], model.model
                with torch.no_grad():
                    x = m.embed_tokens(b.tokens[None])
                    h = lay.input_layernorm(x)
                    at, mlp = lay.self_attn, lay.mlp
                    qkv = at.qkv_proj(h).view(1, T, heads + 2 * kv, dim)
                    gu = mlp.gate_up_proj(h)
                    act = F.swiglu(gu)
                    o = torch.randn(1, T, heads * dim, device="cuda").bfloat16()

                    def ng(f):
                        def run():
                            with torch.no_grad():
                                f()
                        return run

                    add(family, phase, "embedding", ng(lambda: F.embedding(b.tokens, m.embed_tokens.weight)), 0, T * hidden * 4)
                    add(family, phase, "rmsnorm + residual", ng(lambda: lay.input_layernorm(x, h)), 0, T * hidden * 8)
                    gemm("qkv_proj", h, at.qkv_proj.weight, ng(lambda: at.qkv_proj(h)))
                    add(family, phase, "rope", ng(lambda: at.rope(qkv, positions=b.positions, n_rot_heads=heads + kv)), 0, 4 * T * (heads + kv) * dim)
                    add(family, phase, "kv_append", ng(lambda: cache.append(0, qkv[0, :, heads:heads + kv], qkv[0, :, heads + kv:], b.positions, b.slots)),
                        0, 4 * T * 2 * kv * dim)
                    add(family, phase, "attention (paged)", ng(lambda: cache.attend(0, qkv[0, :, :heads], b)), att_flops, att_bytes)
                    if phase == "prefill":
                        q4 = qkv.view(per, prompt, heads + 2 * kv, dim)
                        add(family, phase, "attention (contiguous flash)", ng(lambda: F.flash_attn_fwd(
                            q4[:, :, :heads], q4[:, :, heads:heads + kv], q4[:, :, heads + kv:], True, return_lse=False)), att_flops, att_bytes)
                    gemm("o_proj", o, at.o_proj.weight, ng(lambda: at.o_proj(o)))
                    gemm("gate_up_proj", h, mlp.gate_up_proj.weight, ng(lambda: mlp.gate_up_proj(h)))
                    add(family, phase, "swiglu", ng(lambda: F.swiglu(gu)), 0, T * ff * 6)
                    gemm("down_proj", act, mlp.down_proj.weight, ng(lambda: mlp.down_proj(act)))
                    if phase == "decode":
                        gemm("head", h, model.lm_head.weight, ng(lambda: model.lm_head(h)))
        del model, cache
        gc.collect()
        torch.cuda.empty_cache()
    assert lib.ft_read_device_status(0) == 0, "a kernel reported a timed-out wait"
    return rows


def _zolorax_kernels(add, gemm, model, cache, b, prefill: bool, sizes: tuple) -> None:
    """The kernels of a recurrent, an attention, a dense and a routed sublayer."""
    from ferrotorch_b200.ops import decoder as D
    from ferrotorch_b200.ops import functional as F

    hidden, heads, kv, dim, prompt, per, batch = sizes
    T, dt = b.n_rows, torch.bfloat16
    rec, att, routed = model.layers[0], model.layers[2], model.layers[1]
    C = rec.mixer.spec.padded_width
    x, h = rec.norm1.gather(b.tokens, model.embed, dt)
    add("embedding + norm", lambda: rec.norm1.gather(b.tokens, model.embed, dt), 0, T * hidden * 8)
    add("rms norm", lambda: rec.norm1(x, out_dtype=dt), 0, T * hidden * 6)
    # recurrent mixer
    m, st = rec.mixer, cache.states[0]
    packed = F.linear_rows(h, m.in_proj, m.in_bias)
    y, cx = packed[:, :C], packed[:, C:]
    gemm("recurrent in_proj (y|x) + bias", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj, m.in_bias))
    add("causal conv", lambda: D.causal_conv(cx, m.conv_weight, m.conv_bias, st.conv, b), 0, 4 * T * C)
    u = D.causal_conv(cx, m.conv_weight, m.conv_bias, st.conv, b)
    out = torch.empty((T, C), device="cuda", dtype=dt)
    n, a, z = m.gates.shape[-1], torch.rand((T, C), device="cuda"), torch.randn((T, C), device="cuda")

    def gates():                                          # the portions left out: product and gates alone
        spans, b.spans = b.spans, []
        D.gated_recurrence(u, y, m.gates, m.r_bias, m.i_bias, m.decay, st.state, b, cx, st.conv, out)
        b.spans = spans

    add("gates" + ("" if prefill else " + step"), gates, 4 * T * C * n, 10 * T * C if prefill else 14 * T * C + 2 * m.gates.numel())
    if prefill:
        add("scan * gelu", lambda: D.rglru_scan(a, z, y, out, st.state, b, cx, st.conv), 0, 12 * T * C)
    gemm("recurrent out_proj + residual", out, m.out_proj, lambda: F.residual_linear_(x, out, m.out_proj))
    # attention mixer
    m, s = att.mixer, att.mixer.attn
    (qo, qn), (ko, kn), (vo, vn), (go, gn) = m.segments
    packed = F.linear_rows(h, m.in_proj)
    gemm("attention in_proj (q|k|v|g)", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj))
    add("head norms, rotation, append", lambda: D.qkv_head_finish(
        packed, cache, 0, b, heads=heads, dim=dim, q_off=qo, k_off=ko, v_off=vo, q_weight=m.q_norm, k_weight=m.k_norm, eps=m.eps,
        table=cache.rotary_table(s.rotary)), 0, 4 * T * (qn + kn + vn))
    q, gate = packed[:, qo:qo + qn].unflatten(1, (heads, dim)), packed[:, go:go + gn].unflatten(1, (heads, dim))
    o = torch.empty((T, heads, dim), device="cuda", dtype=dt)
    seen = sum(min(i + 1, s.window) for i in range(prompt))
    add("attention (window %d, sink, gated)" % s.window, lambda: cache.attend(0, q, b, s.scale, gate=gate, out=o, window=s.window, sink=m.sink),
        4 * heads * dim * per * seen if prefill else 0,
        2 * T * (3 * heads + 2 * kv) * dim if prefill else batch * min(prompt, s.window) * kv * 2 * dim * 2)
    gemm("attention out_proj + residual", o.flatten(1), m.out_proj, lambda: F.residual_linear_(x, o.flatten(1), m.out_proj))
    # feed-forwards
    m = rec.mlp
    act = F.linear_rows(h, m.up, activation="relu2")
    gemm("dense up + squared relu", h, m.up, lambda: F.linear_rows(h, m.up, activation="relu2"))
    gemm("dense down + residual", act, m.down, lambda: F.residual_linear_(x, act, m.down))
    m = routed.mlp
    E, top, ff = m.spec.experts, m.spec.top, m.spec.ff
    r = D.moe_route(h, m.router, E, top)
    add("routing (logits, choice, sort, gather)", lambda: D.moe_route(h, m.router, E, top), 2 * T * hidden * E, 2 * T * hidden * (1 + top))
    eact = D.grouped_linear(r.sorted, m.gate_up, r, glu="silu", seg_rows=T)
    yt = D.grouped_linear(eact, m.down, r, seg_rows=T)
    add("experts gate|up + silu", lambda: D.grouped_linear(r.sorted, m.gate_up, r, glu="silu", seg_rows=T), 4 * T * top * hidden * ff,
        2 * (m.gate_up.numel() + T * top * (hidden + ff)))
    add("experts down", lambda: D.grouped_linear(eact, m.down, r, seg_rows=T), 2 * T * top * hidden * ff, 2 * (m.down.numel() + T * top * (hidden + ff)))
    add("rms norm + experts' terms", lambda: rec.norm1(x, pending=(yt, r.place), update=True, out_dtype=dt), 0, T * hidden * (10 + 2 * top))
    if not prefill:
        gemm("head", h, model.head, lambda: F.linear_f32_out(h, model.head))


def _tenalorn_kernels(add, gemm, model, cache, b, prefill: bool, sizes: tuple) -> None:
    """The kernels of a parallel and a latent mixer, the routed feed-forward and the streams."""
    from ferrotorch_b200 import _native
    from ferrotorch_b200.nn.latent_attention import FORMED_PAGE
    from ferrotorch_b200.nn.paged import prefill_pages
    from ferrotorch_b200.ops import decoder as D
    from ferrotorch_b200.ops import functional as F

    hidden, heads, kv, dim, prompt, per, batch = sizes
    T, dt, c = b.n_rows, torch.bfloat16, model.config
    S, par, lat = c.streams, model.layers[0], model.layers[1]

    def embed():
        return D.embed_bigram(b, cache, model.embed, model.bigram, c.embedding_scale, c.bigram.mul_prev, c.bigram.mul_cur, par.hc1.into, par.norm1.weight,
                              c.norm_eps, count=hidden, out_dtype=dt)

    x, h = embed()
    add("embedding + bigram + norm", embed, 0, T * hidden * 10)
    # attention beside memories
    m, a, w = par.mixer, par.mixer.attn, par.mixer.memory
    at = m.offsets
    packed, z = F.linear_rows(h, m.in_proj), D.few_outputs(h, m.gate_proj)
    gemm("parallel in_proj (q|k|v|q'|k'|v'|g')", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj))
    add("memory gates' product (fp32 out)", lambda: D.few_outputs(h, m.gate_proj), 0, 2 * T * hidden)
    add("head norms, append", lambda: D.qkv_head_finish(packed, cache, 0, b, heads=heads, dim=dim, q_off=at["left.q"], k_off=at["left.k"], v_off=at["left.v"],
                                                        q_weight=m.ones, k_weight=m.ones, true_dim=dim, eps=m.eps), 0, 4 * T * (heads + 2 * kv) * dim)
    both = torch.empty((T, m.left_width + m.right_width), device="cuda", dtype=dt)
    q, o = packed[:, at["left.q"]:at["left.k"]].unflatten(1, (heads, dim)), both[:, :m.left_width].unflatten(1, (heads, dim))
    seen = sum(i % a.chunk + 1 for i in range(prompt))
    now = (prompt - 1) % a.chunk + 1
    add("attention (chunks of %d, distance bias)" % a.chunk, lambda: cache.attend(0, q, b, a.scale, out=o, chunk=a.chunk, slopes=m.slopes, out_scale=1.2),
        4 * heads * dim * per * seen if prefill else 0, 2 * T * (2 * heads + 2 * kv) * dim if prefill else batch * now * kv * 2 * dim * 2)

    def memory():
        D.matrix_memory(packed[:, at["right.q"]:at["right.k"]], packed[:, at["right.k"]:at["right.v"]], packed[:, at["right.v"]:at["right.g"]],
                        packed[:, at["right.g"]:], z, m.i_bias, m.f_bias, m.norm, cache.states[0], b, both[:, m.left_width:], heads=w.heads, dim=w.dim,
                        vdim=w.vdim, cap=w.gate_cap, eps=m.eps)

    inner = w.heads * (2 * w.dim + 3 * w.vdim) * 2 * T
    flops = T * w.heads * (2 * 64 * (w.dim + w.vdim) + 4 * w.dim * w.vdim)
    add("matrix memories" + (" (four passes)" if prefill else " (step)"), memory, flops if prefill else 0,
        inner + (0 if prefill else 8 * T * w.heads * w.dim * (w.vdim + 1)))
    gemm("parallel out_proj", both, m.out_proj, lambda: F.linear_rows(both, m.out_proj))
    # latent attention
    m, s = lat.mixer, lat.mixer.spec
    packed = F.linear_rows(h, m.in_proj)
    gemm("latent in_proj (q|latent|g)", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj))
    table, gate = cache.rotary_table(s.rotary), packed[:, m.q_width + s.row_size:]
    q_lat = torch.randn((0 if prefill else T, s.heads, s.row_size), device="cuda").to(dt)
    add("latent norm, rotation, append", lambda: D.latent_finish(
        packed, cache, 1, b, heads=s.heads, q_off=0, q_head=s.head_size, q_rot=s.padded_dim, c_off=m.q_width, rank=s.rank, rank_pad=s.padded_rank,
        weight=m.latent_norm, eps=m.eps, table=table, q_lat=q_lat), 0, 4 * T * (s.row_size + s.heads * s.padded_rot))
    out = torch.empty((T, m.value_width), device="cuda", dtype=dt)
    if prefill:
        rows, spans, longest, pages, items = b.contexts(int(_native.kernels().ft_paged_prefill_tile(1)), FORMED_PAGE)[0]
        ctx = torch.empty((rows, s.row_size), device="cuda", dtype=dt)
        add("latent rows of the contexts", lambda: cache.gather_contexts(1, spans, longest, ctx, FORMED_PAGE), 0, 4 * ctx.numel())
        k, v = F.linear_rows(ctx, m.key_proj), F.linear_rows(ctx, m.value_proj)
        gemm("keys from latents", ctx, m.key_proj, lambda: F.linear_rows(ctx, m.key_proj))
        gemm("values from latents", ctx, m.value_proj, lambda: F.linear_rows(ctx, m.value_proj))
        q4, g4, o4 = (t.unflatten(1, (s.heads, -1)) for t in (packed[:, :m.q_width], gate, out))
        k, v = k.view(-1, FORMED_PAGE, s.heads, s.head_size), v.view(-1, FORMED_PAGE, s.heads, s.padded_vdim)
        add("attention (formed keys, gated)", lambda: prefill_pages(q4, k, v, pages, items, s.scale, out=o4, gate=g4),
            2 * s.heads * (s.head_size + s.padded_vdim) * per * prompt * (prompt + 1) // 2, 2 * T * s.heads * (2 * s.head_size + 3 * s.padded_vdim))
    else:
        add("queries into the latent space", lambda: D.block_linear(packed[:, :m.q_width], m.to_latent, q_lat.flatten(1), a_col=s.head_size, out_col=s.row_size),
            2 * T * m.to_latent.numel(), 2 * (m.to_latent.numel() + T * s.heads * (s.padded_dim + s.padded_rank)))
        o_lat = cache.decode(1, q_lat, b.visible, s.scale, seq_ids=b.slots)
        add("attention (latent rows)", lambda: cache.decode(1, q_lat, b.visible, s.scale, seq_ids=b.slots), 2 * s.heads * (s.row_size + s.padded_rank) * batch * prompt,
            batch * prompt * s.row_size * 2)
        add("values from latents, gated", lambda: D.block_linear(o_lat.flatten(1), m.to_value, out, gate=gate), 2 * T * m.to_value.numel(),
            2 * (m.to_value.numel() + T * s.heads * (s.padded_rank + 2 * s.padded_vdim)))
    gemm("latent out_proj", out, m.out_proj, lambda: F.linear_rows(out, m.out_proj))
    # feed-forward and streams
    m, e = par.mlp, par.mlp.spec
    n_act = T * e.top
    kw = dict(identity=e.identity, score=e.score, correction=m.correction, normalize=e.normalize)
    r = D.moe_route(h, m.router, e.experts, e.top, **kw)
    add("routing (logits, choice, sort, gather)", lambda: D.moe_route(h, m.router, e.experts, e.top, **kw), 2 * T * hidden * e.outputs, 2 * T * hidden * (1 + e.top))
    act = D.grouped_linear(r.sorted, m.gate_up, r, glu="silu", seg_rows=T, scaled=False)
    yt = D.grouped_linear(act, m.down, r, seg_rows=T)
    add("experts gate|up + silu", lambda: D.grouped_linear(r.sorted, m.gate_up, r, glu="silu", seg_rows=T, scaled=False), 4 * n_act * hidden * e.ff,
        2 * (m.gate_up.numel() + n_act * (hidden + e.ff)))
    add("experts down", lambda: D.grouped_linear(act, m.down, r, seg_rows=T), 2 * n_act * hidden * e.ff, 2 * (m.down.numel() + n_act * (hidden + e.ff)))
    act = torch.empty((T, m.shared_down.shape[1]), device="cuda", dtype=dt)
    add("shared expert gate|up + silu", lambda: D.block_linear(h, m.shared_gate_up, act, glu="silu"), 4 * T * hidden * e.shared_ff,
        2 * (m.shared_gate_up.numel() + T * (hidden + e.shared_ff)))
    gemm("shared expert down", act, m.shared_down, lambda: F.linear_rows(act, m.shared_down))
    y = F.linear_rows(act, m.shared_down)
    xs = x[:, None].repeat(1, S, 1)
    add("streams + norm (mixer)", lambda: par.hc1.step(xs, D.SublayerTerms(dense=y), par.hc2.into, par.norm2, dt), 0, T * hidden * (8 * S + 4))
    terms = D.SublayerTerms(yt, r.place, r.weight, y)
    add("streams + norm (experts' terms)", lambda: par.hc2.step(xs, terms, lat.hc1.into, lat.norm1, dt), 0, T * hidden * (8 * S + 4 + 2 * e.top))
    if not prefill:
        gemm("head", h, model.head, lambda: F.linear_f32_out(h, model.head))
        logits = F.linear_f32_out(h, model.head)
        add("soft cap", lambda: D.softcap_(logits, 30.0), 0, 8 * logits.numel())


def _mogelix_kernels(add, gemm, model, cache, b, prefill: bool, sizes: tuple) -> None:
    """The kernels of a state-space and an attention mixer, a dense and a routed feed-forward and the sums with their norms."""
    from ferrotorch_b200.ops import decoder as D
    from ferrotorch_b200.ops import functional as F

    hidden, heads, kv, dim, prompt, per, batch = sizes
    T, dt, c = b.n_rows, torch.bfloat16, model.config
    first, att, routed = model.layers[0], model.layers[1], model.layers[1].mlp
    add("embedding", lambda: F.embedding(b.tokens, model.embed), 0, T * hidden * 4)
    h = F.embedding(b.tokens, model.embed)
    # state-space mixer
    m, w, st = first.mixer, first.mixer.spec, cache.states[0]
    C, inner = w.channels, w.padded_inner
    packed, step = F.linear_rows(h, m.in_proj, m.in_bias), D.few_outputs(h, m.step_proj)
    gemm("state-space in_proj (x|B|C|z|gate) + bias", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj, m.in_bias))
    add("step sizes' product (fp32 out)", lambda: D.few_outputs(h, m.step_proj), 0, 2 * T * hidden)
    xbc, z = packed[:, :C], packed[:, C:m.gate_at]
    add("causal conv + silu", lambda: D.causal_conv(xbc, m.conv_weight, m.conv_bias, st.conv, b, silu=True), 0, 4 * T * C)
    u = D.causal_conv(xbc, m.conv_weight, m.conv_bias, st.conv, b, silu=True)
    y = torch.empty((T, inner), device="cuda", dtype=dt)
    args = (u, z, step, m.step_bias, m.rate, m.skip, st.S, b, y)
    flops = T * w.heads * (2 * 64 * (w.state + w.vdim) + 4 * w.state * w.vdim)
    add("state-space heads" + (" (four passes)" if prefill else " (step)"), lambda: D.state_space(*args, heads=w.heads, groups=w.groups), flops if prefill else 0,
        2 * T * (3 * inner + 2 * w.groups * w.state) + 4 * T * w.heads + (0 if prefill else 8 * T * w.heads * w.state * w.vdim))
    add("part norm", lambda: D.part_norm_(y, m.norm, w.norm_groups, m.eps, heads=w.heads, vdim=w.vdim), 0, 4 * T * inner)
    gemm("state-space out_proj", y, m.out_proj, lambda: F.linear_rows(y, m.out_proj))
    dense, gate = F.linear_rows(y, m.out_proj), packed[:, m.gate_at:]
    x = torch.randn((T, hidden), device="cuda")
    add("sum + gate + norm (mixer)", lambda: D.sum_norm(x, D.SublayerTerms(dense=dense), gate, 3.0, first.norm1.weight, 1e-6, count=hidden, out_dtype=dt), 0, T * hidden * 14)
    # attention mixer
    m, s = att.mixer, att.mixer.attn
    (qo, qn), (ko, kn), (vo, vn), _ = m.segments
    packed = F.linear_rows(h, m.in_proj, m.in_bias)
    gemm("attention in_proj (q|k|v|gate) + bias", h, m.in_proj, lambda: F.linear_rows(h, m.in_proj, m.in_bias))
    add("head norms, rotation, append", lambda: D.qkv_head_finish(
        packed, cache, 0, b, heads=heads, dim=dim, q_off=qo, k_off=ko, v_off=vo, q_weight=m.q_norm, k_weight=m.k_norm, eps=m.eps,
        table=cache.rotary_table(s.rotary)), 0, 4 * T * (qn + kn + vn))
    add("means of blocks", lambda: cache.pool_blocks(0, b), 0, 2 * (T if prefill else batch) * 2 * kv * dim * (1 + 1 / s.pool))
    q, o = packed[:, qo:qo + qn].unflatten(1, (heads, dim)), torch.empty((T, heads, dim), device="cuda", dtype=dt)
    seen = sum(min(i + 1, s.window) + max(0, i + 1 - s.window) // s.pool for i in range(prompt))
    now = min(prompt, s.window) + max(0, prompt - s.window) // s.pool
    add("attention (window %d, blocks of %d, sink)" % (s.window, s.pool), lambda: cache.attend(0, q, b, s.scale, out=o, window=s.window, sink=m.sink, pool=s.pool),
        4 * heads * dim * per * seen if prefill else 0, 2 * T * (2 * heads + 2 * kv) * dim if prefill else batch * now * kv * 2 * dim * 2)
    gemm("attention out_proj", o.flatten(1), m.out_proj, lambda: F.linear_rows(o.flatten(1), m.out_proj))
    # feed-forwards
    m = first.mlp
    n = m.down.shape[1]
    packed = F.linear_rows(h, m.up, m.bias)
    gemm("dense up|gate + bias", h, m.up, lambda: F.linear_rows(h, m.up, m.bias))
    add("poly norm", lambda: D.poly_norm(packed[:, :n], m.act, m.eps, count=n), 0, 4 * T * n)
    act = D.poly_norm(packed[:, :n], m.act, m.eps, count=n)
    gemm("dense down", act, m.down, lambda: F.linear_rows(act, m.down))
    m, e = routed, routed.spec
    kw = dict(score=e.score, normalize=e.normalize, bias=m.router_bias, gate=True)
    r = D.moe_route(h, m.router, e.experts, e.top, **kw)
    add("routing (logits, choice, sort, gather)", lambda: D.moe_route(h, m.router, e.experts, e.top, **kw), 2 * T * hidden * e.experts, 2 * T * hidden * (1 + e.top))
    act = D.grouped_linear(r.sorted, m.gate_up, r, seg_rows=T, activation="relu2")
    yt = D.grouped_linear(act, m.down, r, seg_rows=T)
    n_act = T * e.top
    add("experts up + squared relu", lambda: D.grouped_linear(r.sorted, m.gate_up, r, seg_rows=T, activation="relu2"), 2 * n_act * hidden * e.ff,
        2 * (m.gate_up.numel() + n_act * (hidden + e.ff)))
    add("experts down", lambda: D.grouped_linear(act, m.down, r, seg_rows=T), 2 * n_act * hidden * e.ff, 2 * (m.down.numel() + n_act * (hidden + e.ff)))
    up = m.shared_gate_up[0, 0]
    sact = F.linear_rows(h, up, activation="relu2")
    gemm("shared expert up + squared relu", h, up, lambda: F.linear_rows(h, up, activation="relu2"))
    gemm("shared expert down", sact, m.shared_down, lambda: F.linear_rows(sact, m.shared_down))
    gemm("residual gate + bias", h, m.residual_proj, lambda: F.linear_rows(h, m.residual_proj, m.residual_bias))
    terms = D.SublayerTerms(yt, r.place, r.weight, F.linear_rows(sact, m.shared_down), dense_weight=r.gate)
    gate = F.linear_rows(h, m.residual_proj, m.residual_bias)
    add("sum + gate + norm (experts' terms)", lambda: D.sum_norm(x, terms, gate, 3.0, att.norm2.weight, 1e-6, count=hidden, out_dtype=dt), 0, T * hidden * (14 + 2 * e.top))
    if not prefill:
        gemm("head", h, model.head, lambda: F.linear_f32_out(h, model.head))


def run(args, sampler_cls) -> dict:
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    from ferrotorch_b200 import _native

    sizes, families = args.serving_sizes.split(","), tuple(args.serving_families.split(","))
    out = {"metric": "decoder_serving_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": max(3, args.warmup),
           "dtype": "bf16", "data": "synthetic", "weights": "random", "higher_is_better": True, "sizes": {}, "kernels": {}}
    launches = _native.launch_count()
    sampler = sampler_cls(0)
    sampler.start()
    for size in sizes:
        out["sizes"][size] = {}
        for family in families:
            model = build(family, size)
            out["sizes"][size][family] = throughput(model, size, args.steps, max(3, args.warmup))
            del model
            gc.collect()
            torch.cuda.empty_cache()
        if args.serving_kernels:
            out["kernels"][size] = kernel_table(size, peaks, args.steps, families)
    out["clocks"] = sampler.stop()
    out["gpu_launches"] = _native.launch_count() - launches
    out["device_status"] = _native.device_status(0)
    out["value"] = out["sizes"][sizes[-1]][families[-1]]["decode_tok_s"]
    return out

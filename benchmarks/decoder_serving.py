"""Prefill and decode throughput of the decoder families that the serving engine runs, side by side at equal size.

    python bench.py --workload decoder-serving                 # all families and sizes below
    python bench.py --workload decoder-serving --serving-sizes 8b --serving-kernels

Random weights.  Both families run on ``models.serving.PagedStepper``: prefill feeds prompts of ``prompt`` tokens in steps
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
# two-matrix MLP is 1.5 x as wide, so both have the same number of parameters and matrix-product FLOPs.
SIZES = {"1b": (2048, 16, 32, 8, 64, 8192, 128256, 2048, 64),
         "3b": (3072, 28, 24, 8, 128, 8192, 128256, 2048, 64),
         "8b": (4096, 32, 32, 8, 128, 14336, 128256, 2048, 64)}
FAMILIES = ("llama", "bopudra")
PAGE = 16


def build(family: str, size: str, layers: int | None = None):
    hidden, n, heads, kv, dim, ff, vocab, _, _ = SIZES[size]
    n = layers or n
    if family == "bopudra":
        from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM

        return BopudraForCausalLM(BopudraConfig.uniform(vocab, hidden, n, heads, kv, dim, ff * 3 // 2), device="cuda").random_()
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
        st.feed([(s, [7], [0]) for s in slots])

    dec_host_ms = _event_ms(decode, warmup, steps)         # as served: bookkeeping, one upload, replay
    graph = next(iter(st._graphs.values()))[1]
    dec_ms = _event_ms(graph.replay, warmup, steps)
    return {"prefill_tok_s": round(per * prompt / pre_ms * 1e3), "prefill_ms": round(pre_ms, 3), "prefill_tokens_per_step": per * prompt,
            "decode_tok_s": round(batch / dec_ms * 1e3), "decode_ms": round(dec_ms, 3), "decode_step_as_served_ms": round(dec_host_ms, 3),
            "decode_batch": batch, "context": prompt}


def kernel_table(size: str, peaks: dict, steps: int) -> list:
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
    for family in FAMILIES:
        model = build(family, size, layers=2)
        cache = model.make_paged_cache(batch * ((prompt + 16) // PAGE + 1), PAGE, batch, prompt + 16)
        for s in range(batch):
            cache.reserve(s, prompt + 1)
        cache.sync_table()
        per = max(1, 8192 // prompt)
        pre = RaggedBatch([(s, [1] * prompt, 0, [prompt - 1]) for s in range(per)], "cuda")
        dec = RaggedBatch([(s, [1], prompt - 1, [0]) for s in range(batch)], "cuda")
        for phase, b in (("prefill", pre), ("decode", dec)):
            T = b.n_rows
            kvb = batch * prompt * kv * 2 * dim * 2
            att_flops = 4 * heads * dim * per * prompt * (prompt + 1) // 2 if phase == "prefill" else 0
            att_bytes = 4 * T * (heads + kv) * dim if phase == "prefill" else kvb

            def gemm(name, a, w, fn):
                add(family, phase, name, fn, 2 * T * w.shape[0] * w.shape[1], 2 * (w.numel() + a.numel()))

            if family == "bopudra":
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


def run(args, sampler_cls) -> dict:
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    from ferrotorch_b200 import _native

    sizes = args.serving_sizes.split(",")
    out = {"metric": "decoder_serving_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": max(3, args.warmup),
           "dtype": "bf16", "data": "synthetic", "weights": "random", "higher_is_better": True, "sizes": {}, "kernels": {}}
    launches = _native.launch_count()
    sampler = sampler_cls(0)
    sampler.start()
    for size in sizes:
        out["sizes"][size] = {}
        for family in FAMILIES:
            model = build(family, size)
            out["sizes"][size][family] = throughput(model, size, args.steps, max(3, args.warmup))
            del model
            gc.collect()
            torch.cuda.empty_cache()
        if args.serving_kernels:
            out["kernels"][size] = kernel_table(size, peaks, args.steps)
    out["clocks"] = sampler.stop()
    out["gpu_launches"] = _native.launch_count() - launches
    out["device_status"] = _native.device_status(0)
    out["value"] = out["sizes"][sizes[-1]]["bopudra"]["decode_tok_s"]
    return out

"""Small Bopudra configurations with random weights, and the checks that the CPU and the GPU tests share.

Weights are bf16 values (so both number formats start from the same numbers) with norms, temperatures and score scales
that make attention peaky: a single key carries much of a softmax, so a wrong, missing or foreign key shows in the
logits."""
import copy
import json
import os

import torch

import bopudra_oracle as O
from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM
from ferrotorch_b200.models.serving import ContinuousBatcher, PagedStepper

VOCAB = 77


def layer(heads, kv, dim, vdim, ff, coef=0.4, every=7, sharp=2.5):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": sharp / dim ** 0.5,
                                           "q_temp": {"coef": coef, "every": every}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


# sizes that are equal or 1 in ordinary models differ here: key and value heads, layers, groups of 1 / 3 / 5 / 6, odd widths
CASES = {
    "even": dict(width=64, logit_scale=0.75, eps=1e-5, layers=[layer(4, 2, 32, 32, 96), layer(4, 2, 32, 32, 96)]),
    "uneven": dict(width=52, logit_scale=3.0, eps=1e-3, layers=[layer(6, 2, 24, 40, 60, 0.9, 5), layer(5, 1, 12, 20, None, 0.3, 16),
                                                                layer(3, 3, 36, 8, 33, 0.0, 1), layer(6, 1, 72, 100, 50, 0.25, 64)]),
    "one head": dict(width=24, logit_scale=1.0, eps=1e-6, layers=[layer(1, 1, 16, 64, 40, 1.5, 2), layer(2, 1, 80, 16, 17, 0.1, 3)]),
}


def config_dict(case) -> dict:
    c = copy.deepcopy(CASES[case])
    return {"architecture": "Bopudra", "vocab": VOCAB, "width": c["width"], "logit_scale": c["logit_scale"], "norm": {"eps": c["eps"]},
            "layers": c["layers"]}


def random_weights(cfg: dict, seed: int = 0) -> dict:
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).bfloat16()

    def norm(out, name):
        out[name], out[name + ".b"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.2)
        out[name + ".alpha"] = (torch.rand((), generator=g) * 0.8 + 0.4).bfloat16()

    out = {"embed": rnd(V, W), "head": rnd(V, W, std=W ** -0.5)}
    norm(out, "final.norm")
    for i, entry in enumerate(cfg["layers"]):
        m, pre = entry["mixer"], "l%d." % i
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(out, pre + "norm1")
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv), ("g", H)):
            out[pre + "mix." + n] = rnd(rows, W, std=W ** -0.5)
        out[pre + "mix.o"] = rnd(W, H * Dv, std=1.5 * (H * Dv) ** -0.5)
        out[pre + "mix.q.norm"], out[pre + "mix.k.norm"] = rnd(H * D, std=0.2, mean=1.0), rnd(G * D, std=0.2, mean=1.0)
        if entry["mlp"]:
            ff = entry["mlp"]["ff"]
            out[pre + "mlp.up"], out[pre + "mlp.down"] = rnd(ff, W, std=W ** -0.5), rnd(W, ff, std=ff ** -0.5)
    return out


class Case:
    """A configuration, its weights, the framework's model of them and the oracle's logits (kept per token list)."""

    def __init__(self, name: str, dtype=torch.float32, device="cpu", seed: int = 0):
        self.cfg = config_dict(name)
        self.weights = random_weights(self.cfg, seed)
        self.model = BopudraForCausalLM(BopudraConfig.from_dict(self.cfg), dtype, device)
        self.model.load_tensors(self.weights)
        self.device, self.dtype = device, dtype
        # relative RMS error of a row of logits
        self.tolerance = 3e-5 if dtype == torch.float32 else 0.04
        self._known: dict = {}

    def oracle(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._known:
            for longer, rows in self._known.items():
                if longer[:len(key)] == key:              # causal: a prefix has the same logits
                    return rows[:len(key)]
            self._known[key] = O.forward(self.cfg, self.weights, tokens)
        return self._known[key]

    def check(self, got: torch.Tensor, want: torch.Tensor, what: str = "") -> None:
        got = got.double().cpu()
        assert got.shape == want.shape and bool(torch.isfinite(got).all()), what
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        worst = float(err.max())
        assert worst < self.tolerance, "%s: relative error %.3g at row %d" % (what, worst, int(err.argmax()))

    def stepper(self, tokens: int, seqs: int = 4, block: int = 16, **kw) -> PagedStepper:
        return PagedStepper(self.model, (tokens + block - 1) // block, block, seqs, tokens + block, **kw)

    def tokens(self, n: int, seed: int) -> list:
        return torch.randint(0, VOCAB, (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist()

    def save(self, path) -> None:
        from safetensors.torch import save_file

        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.cfg, f)
        save_file({k: v.contiguous() for k, v in self.weights.items()}, os.path.join(path, "model.safetensors"))


def check_whole_prompt(case: Case) -> None:
    toks = case.tokens(45, 1)
    case.check(feed_all(case, [45], toks), case.oracle(toks), "whole prompt")


def feed_all(case: Case, cuts: list, toks: list, block: int = 16, **kw) -> torch.Tensor:
    """All logits of ``toks`` fed in portions of the sizes ``cuts`` (the last repeated)."""
    st = case.stepper(len(toks), block=block, **kw)
    slot, at, rows, i = st.admit(), 0, [], 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        rows.append(st.feed([(slot, toks[at:at + n], range(n))]).clone())
        at, i = at + n, i + 1
    st.release(slot)
    assert st.manager.free_pages == st.cache.num_blocks
    return torch.cat(rows)


def check_portions(case: Case, block: int = 16, length: int = 75) -> None:
    """Portions of several sizes, single tokens, and mixtures of both give the oracle's logits at every position."""
    toks = case.tokens(length, 2)
    want = case.oracle(toks)
    for cuts in ([2], [1], [length - 9, 1], [3, 1, 16, 2, 1, 1, 17, 5], [16], [33]):
        case.check(feed_all(case, cuts, toks, block), want, "portions %s, pages of %d" % (cuts, block))


def check_batches(case: Case, **kw) -> None:
    """Unequal requests in one batch, admitted, left out, ended and replaced at different steps, in a pool that fits them
    exactly: every logit equals the request's own."""
    reqs = {"a": case.tokens(50, 3), "b": case.tokens(7, 4), "c": case.tokens(33, 5), "d": case.tokens(1, 6), "e": case.tokens(64, 7)}
    steps = [  # (request, tokens) per step
        [("a", 20)], [("b", 1), ("a", 2), ("c", 13)], [("c", 1), ("a", 1), ("b", 1)], [("b", 5), ("d", 1), ("a", 1)],
        [("c", 2), ("a", 16)], [("e", 17), ("a", 1), ("c", 1)], [("a", 9), ("e", 1)], [("e", 2), ("c", 16)], [("e", 1), ("b2", 1)],
        [("b2", 6), ("e", 40), ("d2", 1)], [("e", 1)], [("a2", 50), ("e", 1)], [("e", 1)]]
    st = case.stepper(16 * 12, **kw)
    slots, at, seen_slots = {}, {}, []
    for step in steps:
        parts, rows = [], []
        for rid, n in step:
            toks = reqs[rid[0]]
            if rid not in slots:
                slots[rid] = st.admit()
                seen_slots.append(slots[rid])
            lo = at.get(rid, 0)
            want = [i for i in range(n) if (lo + i) % 3 != 1] if n > 2 else list(range(n))
            parts.append((slots[rid], toks[lo:lo + n], want))
            rows += [case.oracle(toks)[lo + w] for w in want]
            at[rid] = lo + n
        case.check(st.feed(parts), torch.stack(rows), "step %s" % step)
        for rid, _ in step:
            if at[rid] == len(reqs[rid[0]]):
                st.release(slots[rid])
    assert len(set(seen_slots)) < len(seen_slots)         # slots, and with them pages, were used again
    assert st.manager.free_pages == st.cache.num_blocks and st.manager.num_sequences() == 0


def greedy(case: Case, prompt: list, n: int) -> list:
    """The oracle's greedy continuation and the smallest gap between its two best logits."""
    toks, gap = list(prompt), float("inf")
    for _ in range(n):
        z = O.forward(case.cfg, case.weights, toks)[-1]
        top = z.topk(2).values
        gap = min(gap, float(top[0] - top[1]))
        toks.append(int(z.argmax()))
    return toks[len(prompt):], gap


def check_generation(case: Case, blocks: int = 64, n: int = 8, **kw) -> ContinuousBatcher:
    """Greedy generation through the scheduler equals the oracle's, request by request."""
    prompts = [case.tokens(k, 20 + k) for k in (5, 23, 1, 18)]
    want = [greedy(case, p, n) for p in prompts]
    b = ContinuousBatcher(case.model, num_blocks=blocks, block_size=8, max_running=3, max_seq_len=64, prefill_chunk=8, watermark=0.0, **kw)
    reqs = [b.submit(p, n) for p in prompts]
    b.run()
    for r, (tokens, gap) in zip(reqs, want):
        if gap > (1e-3 if case.dtype == torch.float32 else 0.5):      # no near-tie that rounding may turn over
            assert r.output == tokens
    assert all(len(r.output) == n for r in reqs) and b.manager.free_pages == blocks
    return b

"""Checks that the decoder families share: a small model with random weights on the framework's step function, cache and
scheduler against a plain oracle of it."""
import json
import os

import torch

from ferrotorch_b200.models.serving import ContinuousBatcher, PagedStepper

VOCAB = 77


class DecoderCase:
    """A configuration, its weights, the framework's model of them and the oracle's logits (kept per token list).
    ``oracle_forward(cfg, weights, tokens)`` gives the logits ``[T, vocab]``."""

    def __init__(self, cfg: dict, weights: dict, model, oracle_forward):
        self.cfg, self.weights, self.model, self.oracle_forward = cfg, weights, model, oracle_forward
        self.model.load_tensors(self.weights)
        self.device, dtype = model.embed.device, model.dtype
        self.dtype = dtype
        # relative RMS error of a row of logits, and the share of rows that may be over it
        self.loose_rows = 0.0
        self.tolerance = 3e-5 if dtype == torch.float32 else 0.04
        self._known: dict = {}

    def oracle(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._known:
            for longer, rows in self._known.items():
                if longer[:len(key)] == key:              # causal: a prefix has the same logits
                    return rows[:len(key)]
            self._known[key] = self.oracle_forward(self.cfg, self.weights, tokens)
        return self._known[key]

    def check(self, got: torch.Tensor, want: torch.Tensor, what: str = "") -> None:
        got = got.double().cpu()
        assert got.shape == want.shape and bool(torch.isfinite(got).all()), what
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        worst = float(err.max())
        over = int((err >= self.tolerance).sum())
        assert over <= self.loose_rows * len(err) and (over == 0 or worst < 6 * self.tolerance), \
            "%s: relative error %.3g at row %d, %d of %d rows over" % (what, worst, int(err.argmax()), over, len(err))

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


def check_whole_prompt(case: DecoderCase) -> None:
    toks = case.tokens(45, 1)
    case.check(feed_all(case, [45], toks), case.oracle(toks), "whole prompt")


def feed_all(case: DecoderCase, cuts: list, toks: list, block: int = 16, **kw) -> torch.Tensor:
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


def check_portions(case: DecoderCase, block: int = 16, length: int = 75) -> None:
    """Portions of several sizes, single tokens, and mixtures of both give the oracle's logits at every position."""
    toks = case.tokens(length, 2)
    want = case.oracle(toks)
    for cuts in ([2], [1], [length - 9, 1], [3, 1, 16, 2, 1, 1, 17, 5], [16], [33]):
        case.check(feed_all(case, cuts, toks, block), want, "portions %s, pages of %d" % (cuts, block))


def check_batches(case: DecoderCase, **kw) -> None:
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


def greedy(case: DecoderCase, prompt: list, n: int) -> list:
    """The oracle's greedy continuation and the smallest gap between its two best logits."""
    toks, gap = list(prompt), float("inf")
    for _ in range(n):
        z = case.oracle_forward(case.cfg, case.weights, toks)[-1]
        top = z.topk(2).values
        gap = min(gap, float(top[0] - top[1]))
        toks.append(int(z.argmax()))
    return toks[len(prompt):], gap


def check_generation(case: DecoderCase, blocks: int = 64, n: int = 8, **kw) -> ContinuousBatcher:
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

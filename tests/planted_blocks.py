"""Attention over the paged cache with pooled blocks ahead of a window, where one key or one block stands out."""
import torch

import mogelix_oracle as O
from ferrotorch_b200.nn.paged import PagedAttentionManager, PagedKVCache, RaggedBatch


def check_planted_blocks(Hq, Hkv, D, Dv, block, dtype, device, length, window, pool, sink=True, tolerance=None):
    """Keys are noise around a direction of their block; a query is a multiple of one key's or one block mean's direction, whose score
    then stands out by tens.  Targets walk over the first and last key inside the window and those just outside it, the last block
    that is seen, the next one (not seen although its mean may be in the cache), the first block, page and tile borders, and the
    query's own key.  Keys come in portions of several sizes, two sequences at a time with interleaved pages that another
    sequence has used before.  ``sink``: every other head has a sink about as large as the planted score."""
    g = torch.Generator().manual_seed(length + D + pool)
    tol = tolerance or (1e-4 if dtype == torch.float32 else 3e-2)
    pages = (length + block - 1) // block
    cache = PagedKVCache(1, Hkv, D, 2 * pages + 1, 3, length + block, block, device, dtype, v_head_dim=Dv)
    cache.keep_pooled(0, pool)
    cache.keep_pooled(0, pool + 3)                        # two sizes side by side
    mgr = PagedAttentionManager(cache)

    def feed(parts):
        """``(slot, position, keys, values)`` into the cache; the batch."""
        entries = [(s, [0] * len(k), at, []) for s, at, k, _ in parts]
        for s, t, at, _ in entries:
            cache.reserve(s, at + len(t))
        batch = RaggedBatch(entries, device)
        order = [p for p in parts if len(p[2]) == 1] + [p for p in parts if len(p[2]) > 1]
        cache.append(0, torch.cat([p[2] for p in order]).to(device), torch.cat([p[3] for p in order]).to(device), batch.positions, batch.slots)
        cache.pool_blocks(0, batch)
        return batch

    directions = torch.randn(length // pool + 1, Hkv, D, generator=g)
    k = (torch.randn(length, Hkv, D, generator=g) * 0.7 + directions[torch.arange(length) // pool]).to(dtype)
    v = torch.randn(length, Hkv, Dv, generator=g).to(dtype)
    stale = mgr.add_sequence(0)
    feed([(stale, 0, 3.0 * k, 5.0 * v)])
    mgr.remove_sequence(stale)
    other, slot = mgr.add_sequence(0), mgr.add_sequence(0)
    for n in range(1, length + 1, max(1, block - 1)):     # pages of two sequences interleave
        for s in (other, slot):
            cache.reserve(s, min(n + block, length))
    means = torch.stack([k[b * pool:(b + 1) * pool].double().mean(0) for b in range(length // pool)]) if length >= pool else torch.zeros(0, Hkv, D)
    group, scale = Hq // Hkv, 0.25
    q, carried = torch.zeros(length, Hq, D), {}
    for i in range(length):
        seen, first = O.visible_blocks(i, window, pool), max(0, i - window + 1)
        for h in range(Hq):
            c = h // group
            places = [("key", t) for t in (i, first, first - 1, first + 1, i // block * block, i // block * block - 1, 0)]
            places += [("block", b) for b in (seen - 1, seen, 0, seen - 2, seen // 128 * 128, seen // 128 * 128 - 1)]
            kind, t = places[(i * 5 + h * 3) % len(places)]
            if kind == "block" and not 0 <= t < len(means):
                kind, t = "key", i
            t = min(max(t, 0), length - 1)
            kt = means[t, c].float() if kind == "block" else k[t, c].float()
            q[i, h] = kt * (50.0 / scale / kt.pow(2).sum())
            if kind == "block" and t < seen or kind == "key" and first <= t <= i:
                carried[i, h] = means[t, c] if kind == "block" else k[t, c].double()
    q = q.to(dtype)
    sinks = torch.tensor([49.0 if h % 2 else 3.0 for h in range(Hq)]) if sink else torch.full((Hq,), -1e4)
    want = torch.zeros(length, Hq, Dv, dtype=torch.float64)
    for i in range(length):
        for h in range(Hq):
            want[i, h] = O.windowed_attention(q[i, h].double(), k[:i + 1, h // group].double(), v[:i + 1, h // group].double(), scale, sinks[h].double(), i, window, pool)
            if (i, h) in carried:                         # the case is what it claims: what was planted scores by far above zero
                assert float(carried[i, h] @ q[i, h].double()) * scale > 45
    for cuts in ([length], [1], [2, 1, 3, block, 1, pool + 1, 5, window]):
        for kp, vp in cache.pooled.values():              # nothing of an earlier pass
            kp.fill_(20.0), vp.fill_(-9.0)
        at, n = 0, 0
        while at < length:
            step = min(cuts[n % len(cuts)], length - at)
            rows = slice(at, at + step)
            batch = feed([(other, at, -k[rows], -v[rows]), (slot, at, k[rows], v[rows])])
            mine = [r for r, s in enumerate(batch.slots.tolist()) if s == slot]
            buf = torch.zeros(batch.n_rows, Hq * D + 8, dtype=dtype)     # rows lie in a wider buffer, as in a packed projection
            buf[mine, :Hq * D] = q[rows].flatten(1)
            buf = buf.to(device)
            out = torch.full((batch.n_rows, Hq * Dv + 16), 7.0, dtype=dtype, device=device)
            cache.attend(0, buf[:, :Hq * D].unflatten(1, (Hq, D)), batch, scale, window=window, pool=pool, sink=sinks.to(device) if sink else None,
                         out=out[:, :Hq * Dv].unflatten(1, (Hq, Dv)))
            got = out[mine, :Hq * Dv].double().cpu().view(step, Hq, Dv)
            err = (got - want[rows]).abs().amax((1, 2))
            assert float(err.max()) < tol, "cuts %s: error %.3g at position %d" % (cuts, float(err.max()), at + int(err.argmax()))
            assert bool((out[:, Hq * Dv:] == 7.0).all())
            at, n = at + step, n + 1
    if len(means):
        got = cache.gather_pooled(0, pool, slot, len(means))
        assert torch.allclose(got[0].double().cpu(), means, atol=1e-6 if dtype == torch.float32 else 2e-2)

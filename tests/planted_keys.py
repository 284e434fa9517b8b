"""Attention over the paged cache where one key stands out: queries that match exactly one key each."""
import torch

import tenalorn_oracle as TO
import zolorax_oracle as O
from ferrotorch_b200.nn.paged import PagedAttentionManager, PagedKVCache, RaggedBatch


def check_planted_keys(Hq, Hkv, D, Dv, block, dtype, device, length, tolerance=None, window=None, sink=False, elem_gate=False,
                       chunk=None, slopes=None, out_scale=1.0, shared=False):
    """Keys are unit-scale noise; query i is a multiple of one key's direction, so that key's score stands out by tens.
    Targets walk over the first keys, page and tile borders, the query's own key, and the key just after it (which a
    query in a portion must not see although it is in the cache); with a window or chunks also over the keys just inside and
    just outside it.  ``sink``: every other head has a sink about as large as the planted score, the others a small one.
    ``slopes [Hq]``: distance bias.  ``shared``: the values are the leading elements of the keys."""
    g = torch.Generator().manual_seed(length + D)
    tol = tolerance or (1e-4 if dtype == torch.float32 else 3e-2)
    cache = PagedKVCache(1, Hkv, D, 2 * ((length + block - 1) // block) + 3, 3, length + block, block, device, dtype, v_head_dim=Dv,
                         values_in_keys=[shared])
    mgr = PagedAttentionManager(cache)
    other, slot = mgr.add_sequence(0), mgr.add_sequence(0)
    for n in range(1, length + 1, max(1, block - 1)):     # pages of two sequences interleave, not in order
        for s in (other, slot):
            cache.reserve(s, min(n + block, length))
    cache.reserve(slot, length)
    k = torch.randn(length, Hkv, D, generator=g).to(dtype)
    v = k[..., :Dv] if shared else torch.randn(length, Hkv, Dv, generator=g).to(dtype)
    pos = torch.arange(length, dtype=torch.int32, device=device)
    for s, sign in ((other, -1.0), (slot, 1.0)):
        n = cache.lengths[s]
        if shared:
            at = torch.arange(n)
            pages = cache._table_host[s, at // block].long()
            cache.k[0][pages.to(device), (at % block).to(device)] = (sign * k[:n]).to(device)
            continue
        cache.append(0, (sign * k[:n]).to(device), (sign * v[:n]).to(device), pos[:n], torch.full((n,), s, dtype=torch.int32, device=device))
    group, scale = Hq // Hkv, 0.25
    edges = sorted({e for b in (block, 128) for m in range(0, length + b, b) for e in (m - 1, m, m + 1)} | {0, 1, 2, length - 1, length - 2})
    edges = [e for e in edges if 0 <= e < length]
    q, target = torch.zeros(length, Hq, D), {}
    for i in range(length):
        for h in range(Hq):
            near = [i, i + 1] + ([i - window, i - window + 1, i - window - 1, i - window + 2] if window else [])
            near += [i // chunk * chunk + e for e in (0, -1, 1)] if chunk else []
            t = (edges + near)[(i * 7 + h * 3) % (len(edges) + len(near))]
            if (window or chunk) and (i + h) % 3 == 0:
                t = near[(i // 3 + h) % len(near)]
            t = min(max(t, 0), length - 1)
            kt = k[t, h // group].float()
            q[i, h] = kt * (50.0 / scale / kt.pow(2).sum())
            target[i, h] = t
    q = q.to(dtype)
    gate = torch.randn(length, Hq, *([Dv] if elem_gate else []), generator=g).to(dtype)
    sinks = torch.tensor([50.5 if h % 2 else 3.0 for h in range(Hq)]) if sink else None
    want = torch.zeros(length, Hq, Dv, dtype=torch.float64)
    for i in range(length):
        for h in range(Hq):
            c = h // group
            lo, hi = O.visible_keys(i, window)
            lo = max(lo, TO.first_of_chunk(i, chunk)) if chunk else lo
            if slopes is not None:
                o = TO.biased_attention(q[i, h].double(), k[:, c].double(), v[:, c].double(), scale, float(slopes[h]), i, lo) * out_scale
                want[i, h] = o * torch.sigmoid(gate[i, h].double())
                continue
            o = out_scale * O.sink_attention(q[i, h].double(), k[lo:hi, c].double(), v[lo:hi, c].double(), scale, sinks[h].double() if sink else None)
            want[i, h] = o * torch.sigmoid(gate[i, h].double())
            if lo <= target[i, h] < hi and D >= 32 and out_scale == 1.0 and not (sink and h % 2):             # the case is what it claims: that key carries the softmax
                assert (o - v[target[i, h], c].double()).abs().max() < 0.2
    for cuts in ([length], [1], [2, 1, 3, block, 1, 128, 5, 1]):
        entries, at, n = [], 0, 0
        while at < length:
            step = min(cuts[n % len(cuts)], length - at)
            entries.append((slot, [0] * step, at, []))
            at, n = at + step, n + 1
        batch = RaggedBatch(entries, device)
        rows = batch.positions.long().cpu()
        # rows lie in a wider buffer, as in a packed projection
        buf = torch.zeros(length, Hq * D + 8, dtype=dtype)
        buf[:, :Hq * D] = q[rows].flatten(1)
        buf = buf.to(device)
        out = torch.full((length, Hq * Dv + 16), 7.0, dtype=dtype, device=device)
        cache.attend(0, buf[:, :Hq * D].unflatten(1, (Hq, D)), batch, scale, gate=gate[rows].to(device), window=window,
                     sink=sinks.to(device) if sink else None, chunk=chunk, out_scale=out_scale,
                     slopes=slopes.to(device) if slopes is not None else None, out=out[:, :Hq * Dv].unflatten(1, (Hq, Dv)))
        err = (out[:, :Hq * Dv].double().cpu().view(length, Hq, Dv) - want[rows]).abs().amax((1, 2))
        assert float(err.max()) < tol, "cuts %s: error %.3g at position %d" % (cuts, float(err.max()), int(rows[err.argmax()]))
        assert bool((out[:, Hq * Dv:] == 7.0).all())

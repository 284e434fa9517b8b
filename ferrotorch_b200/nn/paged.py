"""Paged KV cache: host-side page bookkeeping + device-side storage consumed by kernels.

Bookkeeping mirrors the reference (ferrotorch-nn/src/paged_attention.rs:155-532): a
``PagePool`` with O(1) allocate / free, a per-sequence page list, and a manager that adds,
extends and drops sequences.  Unlike the reference, the pages are device memory
(``[num_blocks, block_size, n_kv_heads, head_dim]`` for K and for V, per layer) and the block
table is a device tensor read by ``ft_kv_append`` / ``ft_paged_decode`` (``csrc/paged_attn.cu``) and
``ft_paged_prefill`` (``csrc/paged_prefill.cu``).

A forward pass over the cache works on a :class:`RaggedBatch`: any number of sequences, each with any number
of new tokens, as one flat list of rows.  :meth:`PagedKVCache.attend` is its attention.
"""
from __future__ import annotations

import torch

from .. import _native
from ..ops import functional as F
from ..ops import reference as ref

_i, _ll, _f, _vp = _native._i, _native._ll, _native._f, _native._vp
_native.register_protos({
    "ft_kv_append": (_i, [_vp] * 7 + [_i] * 6 + [_ll, _ll, _i, _i, _i, _i, _vp]),
    "ft_paged_decode_scratch": (_ll, [_i, _i, _i, _i]),
    "ft_paged_decode": (_i, [_vp] * 10 + [_i] * 5 + [_ll, _ll, _i, _i, _ll] + [_i, _i, _i, _f, _i, _i] + [_vp] * 2 + [_i, _vp, _f, _i, _i, _vp]),
    "ft_paged_rows": (_i, [_vp] * 9 + [_i] * 5 + [_ll, _ll, _i, _i, _ll] + [_i, _i, _i, _i, _f, _i, _i] + [_vp] * 2 + [_i, _vp, _f, _i, _i, _vp]),
    "ft_pool_blocks": (_i, [_vp] * 7 + [_i] * 5 + [_i] * 5 + [_vp]),
    "ft_latent_decode": (_i, [_vp] * 7 + [_i] * 4 + [_ll, _i, _i, _i, _f, _i, _i, _vp]),
    "ft_latent_gather": (_i, [_vp] * 3 + [_i, _i, _vp] + [_i] * 6 + [_vp]),
    "ft_paged_prefill_tile": (_i, [_i]),
    "ft_paged_prefill": (_i, [_vp] * 8 + [_i] * 6 + [_ll, _ll, _i, _i, _ll] + [_i, _i, _i, _f, _i, _i] + [_vp] * 2 + [_i, _vp, _f, _i, _vp]),
})


def _gate_args(gate: torch.Tensor | None) -> tuple:
    """Row, head and element stride of an output gate ``[T, Hq]`` (one number per head) or ``[T, Hq, Dv]``."""
    if gate is None:
        return 0, 0, 0
    return (gate.stride(0), gate.stride(1), gate.stride(2)) if gate.dim() == 3 else (gate.stride(0), gate.stride(1), 0)


def _ptr(t: torch.Tensor | None):
    return t.data_ptr() if t is not None else None


def _pool_args(pool: int | None, pooled: tuple | None) -> tuple:
    """Pooled keys, pooled values and tokens of a block."""
    return (pooled[0].data_ptr(), pooled[1].data_ptr(), pool) if pool else (None, None, 0)


def prefill_pages(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, table: torch.Tensor, items: torch.Tensor, scale: float, *,
                  out: torch.Tensor, gate: torch.Tensor | None = None, window: int | None = None, sink: torch.Tensor | None = None,
                  chunk: int | None = None, slopes: torch.Tensor | None = None, out_scale: float = 1.0, pool: int | None = None,
                  pooled: tuple | None = None) -> None:
    """Attention of the portions listed in ``items`` (device only): ``q [T, Hq, D]``, pages ``k [pages, tokens, Hkv, D]`` and ``v``,
    block table ``[sequences, pages of one]``; ``pooled``: the pages' pooled keys and values (:meth:`PagedKVCache.keep_pooled`)."""
    T, Hq, D = q.shape
    pages, bs, Hkv, Dv = v.shape
    rc = _native.kernels().ft_paged_prefill(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), table.data_ptr(), items.data_ptr(), _ptr(gate), _ptr(sink), out.data_ptr(), items.shape[0], T, Hq, Hkv, D,
        Dv, q.stride(0), *_gate_args(gate), out.stride(0), bs, table.shape[1], pages, float(scale), int(window or 0), int(chunk or 0), *_pool_args(pool, pooled),
        _ptr(slopes), float(out_scale), F._dev(q), F._stream())
    _native.check(rc, "ft_paged_prefill")


class OutOfPages(RuntimeError):
    pass


class PagePool:
    """Free-list of page ids (paged_attention.rs:155-260) with a reference count per page: a page that several
    sequences share (a common prompt prefix) returns to the free list when its last holder lets go."""

    def __init__(self, num_pages: int):
        self.num_pages = num_pages
        self._free = list(range(num_pages - 1, -1, -1))
        self._refs = [0] * num_pages

    def allocate(self) -> int:
        if not self._free:
            raise OutOfPages("page pool exhausted (%d pages)" % self.num_pages)
        page = self._free.pop()
        self._refs[page] = 1
        return page

    def retain(self, page: int) -> int:
        """One more holder of an allocated page."""
        if not 0 <= page < self.num_pages or self._refs[page] == 0:
            raise ValueError("page %d is not allocated" % page)
        self._refs[page] += 1
        return page

    def ref_count(self, page: int) -> int:
        return self._refs[page]

    def free(self, page: int) -> None:
        if not 0 <= page < self.num_pages:
            raise ValueError("page %d out of range" % page)
        if self._refs[page] == 0:
            raise ValueError("page %d is free already" % page)
        self._refs[page] -= 1
        if self._refs[page] == 0:
            self._free.append(page)

    def alloc_page(self):
        """A free page id, or ``None`` when the pool is exhausted (paged_attention.rs:200; ``allocate`` raises)."""
        return self.allocate() if self._free else None

    free_page = free

    @property
    def num_free(self) -> int:
        return len(self._free)

    @property
    def num_used(self) -> int:
        return self.num_pages - len(self._free)

    @property
    def num_total(self) -> int:
        return self.num_pages


class RaggedBatch:
    """The rows of one forward pass: ``entries`` are ``(slot, tokens, start, want)`` -- a sequence slot, its next
    token ids, the position of the first of them, and the places among them whose logits are asked for.

    Entries of one token come first (:attr:`n_single` rows, the decode kernel's batch), longer ones after them
    (:attr:`spans`, the prefill kernel's portions); ``starts`` holds the first position of every row's entry; ``last``
    lists the wanted rows in the order of the entries as they were given.  Everything the kernels read is copied to the
    device in one transfer."""

    def __init__(self, entries: list, device):
        self.device = torch.device(device)
        order = [i for i, e in enumerate(entries) if len(e[1]) == 1]
        self.n_single = len(order)
        order += [i for i, e in enumerate(entries) if len(e[1]) > 1]
        toks, pos, slots, starts, self.spans, first_row, row = [], [], [], [], [], {}, 0
        for i in order:
            slot, tokens, start, _ = entries[i]
            n = len(tokens)
            first_row[i] = row
            toks += tokens
            pos += range(start, start + n)
            slots += [slot] * n
            starts += [start] * n
            if n > 1:
                self.spans.append((slot, row, start, n))
            row += n
        want = [first_row[i] + w for i, e in enumerate(entries) if len(e[1]) for w in e[3]]
        self.n_rows, self.n_want = row, len(want)
        self._fill(toks, pos, slots, [p + 1 for p in pos], starts, want)
        self._items: dict = {}

    def _fill(self, toks, pos, slots, visible, starts, want) -> None:
        """One buffer: token ids and wanted rows as int64, then positions, slots, visible-key counts, entry starts and
        the portions (slot, first row, first position, tokens) as int32."""
        n, m, k = len(toks), len(want), len(self.spans)
        ints = pos + slots + visible + starts + [v for span in self.spans for v in span]
        host = torch.empty(n + m + (len(ints) + 1) // 2, dtype=torch.long, pin_memory=self.device.type == "cuda")
        host[:n + m] = torch.tensor(toks + want, dtype=torch.long)
        host[n + m:].view(torch.int32)[:len(ints)] = torch.tensor(ints, dtype=torch.int32)
        self._buf = host.to(self.device, non_blocking=True)
        self._host = host                                  # the pinned source lives as long as the batch
        ints = self._buf[n + m:].view(torch.int32)
        self.tokens, self.last = self._buf[:n], self._buf[n:n + m]
        self.positions, self.slots, self.visible, self.starts = ints[:n], ints[n:2 * n], ints[2 * n:3 * n], ints[3 * n:4 * n]
        self.span_table = ints[4 * n:4 * n + 4 * k].view(k, 4)

    @property
    def longest(self) -> int:
        """Tokens of the longest portion."""
        return max((s[3] for s in self.spans), default=0)

    def work_items(self, tile_tokens: int):
        """The portions cut into work items of the prefill kernel (``[n, 4]`` int32 on the device: slot, first row,
        tokens, first position; at most ``2 * tile_tokens`` tokens each), longest key range first."""
        got = self._items.get(tile_tokens)
        if got is None:
            rows, step = [], 2 * tile_tokens
            for slot, row, start, n in self.spans:
                rows += [(slot, row + o, min(step, n - o), start + o) for o in range(0, n, step)]
            rows.sort(key=lambda r: -(r[2] + r[3]))
            host = torch.tensor(rows, dtype=torch.int32)
            got = host.pin_memory().to(self.device, non_blocking=True) if self.device.type == "cuda" else host
            self._items[tile_tokens] = got
        return got


    def contexts(self, tile_tokens: int, page: int = 128, limit: int = 32768) -> list:
        """The portions' contexts laid out one after another in pages of ``page`` rows of their own, for attention over keys that are
        formed for this step: groups ``(rows, spans [n, 3], longest, block table [n, pages], work items [m, 4])`` of at most ``limit``
        rows (a longer context is a group of its own); spans are ``(slot, first row, tokens)``, items as in :meth:`work_items` with
        the place in the group's table instead of the slot."""
        key = ("contexts", tile_tokens, page, limit)
        got = self._items.get(key)
        if got is None:
            got, group, rows = [], [], 0
            for span in self.spans:
                need = (span[2] + span[3] + page - 1) // page * page
                if group and rows + need > limit:
                    got.append(self._context_group(group, rows, tile_tokens, page))
                    group, rows = [], 0
                group.append((*span, rows))
                rows += need
            got.append(self._context_group(group, rows, tile_tokens, page))
            self._items[key] = got
        return got

    def _context_group(self, group: list, rows: int, tile_tokens: int, page: int) -> tuple:
        step, n = 2 * tile_tokens, len(group)
        longest = max(s[2] + s[3] for s in group)
        width = (longest + page - 1) // page
        spans = [v for slot, _, start, k, first in group for v in (slot, first, start + k)]
        table = [min(first // page + j, rows // page - 1) for *_, first in group for j in range(width)]
        items = [(i, row + o, min(step, k - o), start + o) for i, (_, row, start, k, _) in enumerate(group) for o in range(0, k, step)]
        items.sort(key=lambda r: -(r[2] + r[3]))
        host = torch.tensor(spans + table + [v for r in items for v in r], dtype=torch.int32)
        buf = host.pin_memory().to(self.device, non_blocking=True) if self.device.type == "cuda" else host
        a, b = 3 * n, 3 * n + n * width
        return rows, buf[:a].view(n, 3), longest, buf[a:b].view(n, width), buf[b:].view(-1, 4)

    def chunk_table(self, rows: int):
        """The portions cut into chunks of ``rows`` tokens, portion after portion: ``(first chunk of every portion [n_spans], chunks
        [n, 4])``, int32 on the device; a chunk is portion, first row, rows, number within the portion."""
        got = self._items.get(("chunks", rows))
        if got is None:
            first, chunks = [], []
            for i, (_, row, _, n) in enumerate(self.spans):
                first.append(len(chunks))
                chunks += [(i, row + o, min(rows, n - o), o // rows) for o in range(0, n, rows)]
            host = torch.tensor(first + [v for c in chunks for v in c], dtype=torch.int32)
            buf = host.pin_memory().to(self.device, non_blocking=True) if self.device.type == "cuda" else host
            got = self._items[("chunks", rows)] = (buf[:len(first)], buf[len(first):].view(-1, 4), host)
        return got[:2]


class DecodeBatch(RaggedBatch):
    """A batch of single-token rows whose device tensors keep their addresses, for captured decode steps: ``rows``
    rows, of which :meth:`load` fills some; the others belong to no sequence (no visible key, no page)."""

    def __init__(self, rows: int, pad_slot: int, device):
        self.device = torch.device(device)
        self.n_single = self.n_rows = self.n_want = rows
        self.spans, self._items, self.pad_slot = [], {}, pad_slot
        self._fill([0] * rows, [0] * rows, [pad_slot] * rows, [0] * rows, [0] * rows, list(range(rows)))
        self._static = self._buf

    def load(self, tokens: list, positions: list, slots: list) -> None:
        pad = self.n_rows - len(tokens)
        views = (self.tokens, self.last, self.positions, self.slots, self.visible, self.starts, self.span_table)
        self._fill(tokens + [0] * pad, positions + [0] * pad, slots + [self.pad_slot] * pad,
                   [p + 1 for p in positions] + [0] * pad, positions + [0] * pad, list(range(self.n_rows)))
        self._static.copy_(self._buf)
        self._buf = self._static
        self.tokens, self.last, self.positions, self.slots, self.visible, self.starts, self.span_table = views


class PagedKVCache:
    """Block tables for up to ``max_seqs`` sequences over one :class:`PagePool`, plus the device
    K/V pages of every layer.  ``block_size`` tokens per page (16 in the benchmark configs).
    ``n_kv_heads``, ``head_dim`` and ``v_head_dim`` (default: ``head_dim``) are numbers, or one number per layer.

    :meth:`keep_pooled` adds, for a layer, the means of the keys and values of every block of so many consecutive positions.  They lie
    with the page that holds the block's last position, so they move, are shared and are given back with it.

    ``values_in_keys`` (per layer, default none): a layer without values of its own; its values are the leading ``v_head_dim``
    elements of its keys (latent attention).

    ``states``: what layers keep per sequence slot besides keys and values (recurrent states, by layer).  A state holds
    the whole sequence so far, so such a cache cannot take tokens back (:attr:`rewindable`) nor start from shared pages."""

    def __init__(self, n_layers: int, n_kv_heads, head_dim, num_blocks: int, max_seqs: int,
                 max_seq_len: int, block_size: int = 16, device="cuda", dtype=torch.bfloat16, v_head_dim=None,
                 values_in_keys: list | None = None):
        def per_layer(v):
            return [int(v)] * n_layers if isinstance(v, int) else [int(x) for x in v]

        self.shapes = list(zip(per_layer(n_kv_heads), per_layer(head_dim), per_layer(head_dim if v_head_dim is None else v_head_dim)))
        if len(self.shapes) != n_layers:
            raise ValueError("PagedKVCache: %d layer shapes for %d layers" % (len(self.shapes), n_layers))
        self.n_layers, self.dtype = n_layers, dtype
        self.n_kv_heads, self.head_dim = self.shapes[0][:2] if self.shapes else (0, 0)
        self.block_size, self.num_blocks, self.max_seqs = block_size, num_blocks, max_seqs
        self.max_blocks = (max_seq_len + block_size - 1) // block_size
        self.device = torch.device(device)
        self.pool = PagePool(num_blocks)
        self.k = [torch.zeros((num_blocks, block_size, h, d), device=self.device, dtype=dtype) for h, d, _ in self.shapes]
        self.values_in_keys = list(values_in_keys) if values_in_keys is not None else [False] * n_layers
        self.v = [k[..., :dv] if shared else torch.zeros((num_blocks, block_size, h, dv), device=self.device, dtype=dtype)
                  for (h, _, dv), k, shared in zip(self.shapes, self.k, self.values_in_keys)]
        self.token_pages: torch.Tensor | None = None
        self.pooled: dict = {}                            # (layer, tokens of a block): pooled keys, pooled values
        # one row more than there are sequences: the padding rows of a captured decode step own no page
        self.pad_slot = max_seqs
        self._table_host = torch.full((max_seqs + 1, self.max_blocks), -1, dtype=torch.int32)
        self.block_table = self._table_host.to(self.device)
        self._pages: list[list[int]] = [[] for _ in range(max_seqs)]
        self.lengths = [0] * max_seqs
        self._dirty = False
        self.states: dict = {}
        self._rotary: dict = {}

    def rotary_table(self, spec) -> torch.Tensor:
        """The table of a :class:`~ferrotorch_b200.nn.packed_block.RotarySpec` for every position the cache can hold."""
        got = self._rotary.get(spec)
        if got is None:
            got = self._rotary[spec] = spec.table(self.max_blocks * self.block_size, self.device)
        return got

    def keep_tokens(self) -> None:
        """Also keep the token of every position in the pages (for embeddings that look back)."""
        self.token_pages = torch.zeros((self.num_blocks, self.block_size), device=self.device, dtype=torch.int32)

    def keep_pooled(self, layer: int, pool: int) -> None:
        """Also keep the means of every block of ``pool`` positions (counted from 0) of a layer: ``[pages, blocks that can end in a
        page, heads, size]``.  Block b is number ``b - first position of its page // pool`` of the page that holds its last position."""
        if self.values_in_keys[layer]:
            raise ValueError("PagedKVCache.keep_pooled: layer %d has no values of its own" % layer)
        if (layer, pool) not in self.pooled:
            h, d, dv = self.shapes[layer]
            per = (self.block_size - 1) // pool + 1
            self.pooled[layer, pool] = tuple(torch.zeros((self.num_blocks, per, h, n), device=self.device, dtype=self.dtype) for n in (d, dv))

    def _pooled_places(self, slots: torch.Tensor, blocks: torch.Tensor, pool: int) -> tuple:
        """Page and place in it of pooled blocks of sequences (host path)."""
        page = (blocks * pool + pool - 1) // self.block_size
        return self._table_host[slots, page].long().clamp(min=0), blocks - page * self.block_size // pool

    def pool_blocks(self, layer: int, batch: RaggedBatch) -> None:
        """The means of the blocks that end among the rows of a batch, whose keys and values the layer's pages already hold."""
        for (at, pool), (kp, vp) in self.pooled.items():
            if at != layer:
                continue
            if self.device.type != "cuda":
                pos, slots = batch.positions.long(), batch.slots.long()
                ends = ((pos + 1) % pool == 0) & (batch.visible > 0)
                pos, slots = pos[ends], slots[ends]
                known = pos[:, None] + torch.arange(1 - pool, 1)
                pages = self._table_host[slots[:, None], known // self.block_size].long()
                place = self._pooled_places(slots, pos // pool, pool)
                for src, dst in ((self.k[layer], kp), (self.v[layer], vp)):
                    dst[place] = src[pages, known % self.block_size].float().mean(1).to(dst.dtype)
                continue
            h, d, dv = self.shapes[layer]
            rc = _native.kernels().ft_pool_blocks(
                self.k[layer].data_ptr(), self.v[layer].data_ptr(), kp.data_ptr(), vp.data_ptr(), self.sync_table().data_ptr(), batch.positions.data_ptr(),
                batch.slots.data_ptr(), batch.n_rows, h, d, dv, pool, int(self.dtype == torch.float32), self.block_size, self.max_blocks, self.num_blocks,
                F._dev(kp), F._stream())
            _native.check(rc, "ft_pool_blocks")

    def gather_pooled(self, layer: int, pool: int, seq: int, blocks: int):
        """Contiguous ``[blocks, Hkv, D]`` pooled keys and ``[blocks, Hkv, Dv]`` values of one sequence (reference path)."""
        b = torch.arange(blocks)
        place = self._pooled_places(torch.full_like(b, seq), b, pool)
        return tuple(t[place] for t in self.pooled[layer, pool])

    @property
    def rewindable(self) -> bool:
        """Whether a sequence can drop its latest tokens or adopt a prefix: yes while pages are all it has."""
        return not self.states

    # ------------------------------------------------------------------ bookkeeping (host)
    def reserve(self, seq: int, new_len: int) -> None:
        """Make sure sequence ``seq`` has pages for ``new_len`` tokens."""
        need = (new_len + self.block_size - 1) // self.block_size
        if need > self.max_blocks:
            raise ValueError("sequence length %d exceeds max_seq_len" % new_len)
        pages = self._pages[seq]
        while len(pages) < need:
            p = self.pool.allocate()
            self._table_host[seq, len(pages)] = p
            pages.append(p)
            self._dirty = True
        self.lengths[seq] = max(self.lengths[seq], new_len)

    def adopt(self, seq: int, pages: list, length: int) -> None:
        """Start sequence ``seq`` on pages that already hold its first ``length`` tokens (whole pages that
        another sequence filled; every one gains a holder).  The sequence must be empty."""
        if not self.rewindable:
            raise ValueError("adopt: recurrent states do not come with the pages of a prefix")
        if self._pages[seq]:
            raise ValueError("adopt: sequence %d already has pages" % seq)
        if length != len(pages) * self.block_size or len(pages) > self.max_blocks:
            raise ValueError("adopt: %d pages of %d tokens cannot hold a prefix of %d" % (len(pages), self.block_size, length))
        for i, p in enumerate(pages):
            self._table_host[seq, i] = self.pool.retain(p)
        self._pages[seq] = list(pages)
        self.lengths[seq] = length
        self._dirty = bool(pages) or self._dirty

    def pages_of(self, seq: int) -> list:
        return list(self._pages[seq])

    def free_sequence(self, seq: int) -> None:
        for p in self._pages[seq]:
            self.pool.free(p)
        self._pages[seq] = []
        self._table_host[seq].fill_(-1)
        self.lengths[seq] = 0
        self._dirty = True

    def sync_table(self) -> torch.Tensor:
        if self._dirty:
            self.block_table.copy_(self._table_host, non_blocking=True)
            self._dirty = False
        return self.block_table

    # ------------------------------------------------------------------ device ops
    def append(self, layer: int, k_new: torch.Tensor, v_new: torch.Tensor, positions: torch.Tensor,
               seq_ids: torch.Tensor | None = None, tokens_per_seq: int = 1) -> None:
        """Write ``k_new / v_new [T, Hkv, D]`` at ``positions [T]`` (int32).  Token i belongs to
        sequence ``seq_ids[i]`` or ``i // tokens_per_seq``.  Pages must have been reserved."""
        T = k_new.shape[0]
        if self.values_in_keys[layer]:
            raise ValueError("PagedKVCache.append: layer %d has no values of its own" % layer)
        table = self.sync_table()
        Hkv, D, Dv = self.shapes[layer]
        if not k_new.is_cuda:
            sid = (seq_ids if seq_ids is not None else torch.arange(T) // tokens_per_seq).long()
            pos = positions.long()
            blk = self._table_host[sid, pos // self.block_size].long()
            if bool((blk < 0).any()):
                raise ValueError("PagedKVCache.append: a position has no page (reserve the sequence first)")
            self.k[layer][blk, pos % self.block_size] = k_new.to(self.k[layer].dtype)
            self.v[layer][blk, pos % self.block_size] = v_new.to(self.v[layer].dtype)
            return
        if k_new.dtype != self.dtype or v_new.dtype != self.dtype:
            raise ValueError("PagedKVCache.append: the cache holds %s, got %s / %s" % (self.dtype, k_new.dtype, v_new.dtype))
        unit = 16 // k_new.element_size()
        k_new, v_new = (t if t.stride(-1) == 1 and t.stride(1) == t.shape[2] and t.stride(0) % unit == 0 and t.data_ptr() % 16 == 0
                        else t.contiguous() for t in (k_new, v_new))
        ldk = k_new.stride(0)
        ldv = v_new.stride(0)
        rc = _native.kernels().ft_kv_append(
            k_new.data_ptr(), v_new.data_ptr(), self.k[layer].data_ptr(), self.v[layer].data_ptr(),
            table.data_ptr(), positions.data_ptr(), seq_ids.data_ptr() if seq_ids is not None else None, T,
            tokens_per_seq, Hkv, D, Dv, k_new.element_size(), ldk, ldv, self.block_size, self.max_blocks,
            self.num_blocks, F._dev(k_new), F._stream())
        _native.check(rc, "ft_kv_append")

    def _check_pool(self, layer: int, pool, window, chunk, slopes) -> None:
        if pool and (not window or chunk or slopes is not None or (layer, pool) not in self.pooled):
            raise ValueError("PagedKVCache: blocks of %d positions of layer %d are not kept, or come without a window" % (pool, layer))

    def _tensor_core_ok(self, layer: int, q: torch.Tensor, max_group: int) -> bool:
        Hkv, D, Dv = self.shapes[layer]
        return (q.dtype == torch.bfloat16 and not self.values_in_keys[layer] and D % 16 == 0 and Dv % 16 == 0 and D <= 128 and Dv <= 128
                and q.shape[1] // Hkv <= max_group and q.data_ptr() % 16 == 0 and q.stride(0) % 8 == 0)

    def _rows(self, layer: int, q, visible, slots, scale, gate, out, window, sink, chunk=None, slopes=None, out_scale=1.0, pool=None) -> None:
        """Attention of arbitrary rows, any head sizes, bf16 or fp32 (the simple kernel)."""
        T, Hq, D = q.shape
        Hkv, _, Dv = self.shapes[layer]
        rc = _native.kernels().ft_paged_rows(
            q.data_ptr(), self.k[layer].data_ptr(), self.v[layer].data_ptr(), self.block_table.data_ptr(), slots.data_ptr(),
            visible.data_ptr(), _ptr(gate), _ptr(sink), out.data_ptr(), T, Hq, Hkv, D, Dv, q.stride(0),
            *_gate_args(gate), out.stride(0), self.v[layer].stride(2), self.block_size, self.max_blocks, self.num_blocks, float(scale),
            int(window or 0), int(chunk or 0), *_pool_args(pool, self.pooled.get((layer, pool))), _ptr(slopes), float(out_scale),
            int(q.dtype == torch.float32), F._dev(q), F._stream())
        _native.check(rc, "ft_paged_rows")

    def decode(self, layer: int, q: torch.Tensor, ctx_len: torch.Tensor, scale: float | None = None,
               n_splits: int = 0, seq_ids: torch.Tensor | None = None, gate: torch.Tensor | None = None,
               out: torch.Tensor | None = None, window: int | None = None, sink: torch.Tensor | None = None,
               chunk: int | None = None, slopes: torch.Tensor | None = None, out_scale: float = 1.0, pool: int | None = None) -> torch.Tensor:
        """One query token per sequence: ``q [B, Hq, D]``, ``ctx_len [B]`` int32 -> ``[B, Hq, Dv]``.  Row b
        reads sequence b, or sequence ``seq_ids[b]`` (int32; a batch of any subset of the live sequences).
        ``gate [B, Hq]`` or ``[B, Hq, Dv]``: output heads or elements are multiplied by its sigmoid.  ``window``: only the
        last so many keys are visible; ``chunk``: those of the query's own chunk of so many positions, counted from 0.  ``sink
        [Hq]`` (fp32): its exponential joins a head's denominator.  ``slopes [Hq]`` (fp32): times the distance of a key, taken off
        its score.  ``out_scale``: factor of the result.  ``pool`` (with a window): the means of the blocks of so many positions that lie
        wholly ahead of the window are visible too (:meth:`keep_pooled`).  ``out``: where the result goes (the heads of a row packed, any row stride)."""
        B, Hq, D = q.shape
        Hkv, _, Dv = self.shapes[layer]
        scale = scale if scale is not None else D ** -0.5
        table = self.sync_table()
        self._check_pool(layer, pool, window, chunk, slopes)
        if not q.is_cuda:
            o = self._decode_reference(layer, q, ctx_len, scale, seq_ids, window, sink, chunk, slopes, pool)
            o = self._finish_reference(o, gate, out_scale)
            return o if out is None else out.copy_(o)
        if out is None:
            out = torch.empty((B, Hq, Dv), device=q.device, dtype=q.dtype)
        seq_ids = seq_ids.to(device=q.device, dtype=torch.int32) if seq_ids is not None else None
        plain = gate is None and not window and sink is None and not chunk and slopes is None and out_scale == 1.0
        if plain and self._latent_ok(layer, q):
            return self._latent_rows(layer, q, ctx_len, seq_ids, scale, out, n_splits)
        if not self._tensor_core_ok(layer, q, 16) and (q.dtype != torch.bfloat16 or self.values_in_keys[layer] or D != Dv or D not in (64, 128)
                                                       or Hq // Hkv not in (1, 2, 4, 8) or pool):
            rows = seq_ids if seq_ids is not None else torch.arange(B, device=q.device, dtype=torch.int32)
            self._rows(layer, q, ctx_len, rows, scale, gate, out, window, sink, chunk, slopes, out_scale, pool)
            return out
        lib = _native.kernels()
        if n_splits <= 0:
            ctas = B * Hkv
            n_splits = 1 if ctas >= 256 else max(1, min(8, 296 // max(ctas, 1)))
            if window and not pool:
                n_splits = min(n_splits, (window + 126) // 128 + 1)          # tiles of 128 keys that a window can touch
            if chunk:
                n_splits = min(n_splits, (chunk + 126) // 128 + 1)
        n_scr = int(lib.ft_paged_decode_scratch(B, Hq, Dv, n_splits))
        scratch = F._get_scratch("paged_decode", n_scr, q.device) if n_scr else None
        rc = lib.ft_paged_decode(q.data_ptr(), self.k[layer].data_ptr(), self.v[layer].data_ptr(), table.data_ptr(),
                                 seq_ids.data_ptr() if seq_ids is not None else None, ctx_len.data_ptr(),
                                 _ptr(gate), _ptr(sink), out.data_ptr(),
                                 scratch.data_ptr() if scratch is not None else None, B, Hq, Hkv, D, Dv, q.stride(0),
                                 *_gate_args(gate), out.stride(0), self.block_size, self.max_blocks, self.num_blocks,
                                 float(scale), int(window or 0), int(chunk or 0), *_pool_args(pool, self.pooled.get((layer, pool))),
                                 _ptr(slopes), float(out_scale), n_splits, F._dev(q), F._stream())
        _native.check(rc, "ft_paged_decode")
        return out

    def attend(self, layer: int, q: torch.Tensor, batch: RaggedBatch, scale: float | None = None,
               gate: torch.Tensor | None = None, out: torch.Tensor | None = None, window: int | None = None,
               sink: torch.Tensor | None = None, chunk: int | None = None, slopes: torch.Tensor | None = None,
               out_scale: float = 1.0, pool: int | None = None) -> torch.Tensor:
        """Causal attention of a whole :class:`RaggedBatch` (its keys and values already appended): ``q [T, Hq, D]`` ->
        ``[T, Hq, Dv]``.  Single tokens run on the decode kernel, longer portions on the prefill kernel; head sizes or
        types that those do not cover run on the simple kernel.  The other arguments as in :meth:`decode`."""
        T, Hq, D = q.shape
        Hkv, _, Dv = self.shapes[layer]
        scale = scale if scale is not None else D ** -0.5
        if out is None:
            out = torch.empty((T, Hq, Dv), device=q.device, dtype=q.dtype)
        table = self.sync_table()
        self._check_pool(layer, pool, window, chunk, slopes)
        n1 = batch.n_single
        if n1:
            self.decode(layer, q[:n1], batch.visible[:n1], scale, seq_ids=batch.slots[:n1],
                        gate=gate[:n1] if gate is not None else None, out=out[:n1], window=window, sink=sink, chunk=chunk, slopes=slopes,
                        out_scale=out_scale, pool=pool)
        if not batch.spans:
            return out
        if not q.is_cuda:
            for slot, row, start, n in batch.spans:
                k, v = self.gather(layer, slot, start + n)
                kp, vp = self.gather_pooled(layer, pool, slot, max(0, start + n - window) // pool) if pool else (k[:0], v[:0])
                o = ref.attention(q[None, row:row + n], k[None], v[None], True, scale, start, window, sink, chunk, slopes, pool, (kp[None], vp[None]))[0][0]
                out[row:row + n] = self._finish_reference(o, gate[row:row + n] if gate is not None else None, out_scale)
            return out
        bs = self.block_size
        if self.values_in_keys[layer]:                    # a portion's rows are as good as single ones
            self.decode(layer, q[n1:], batch.visible[n1:], scale, seq_ids=batch.slots[n1:], gate=gate[n1:] if gate is not None else None, out=out[n1:],
                        window=window, sink=sink, chunk=chunk, slopes=slopes, out_scale=out_scale)
            return out
        if not (self._tensor_core_ok(layer, q, 128) and scale > 0 and bs >= 8 and (128 % bs == 0 or bs % 128 == 0)):
            self._rows(layer, q[n1:], batch.visible[n1:], batch.slots[n1:], scale, gate[n1:] if gate is not None else None, out[n1:],
                       window, sink, chunk, slopes, out_scale, pool)
            return out
        items = batch.work_items(int(_native.kernels().ft_paged_prefill_tile(Hq // Hkv)))
        prefill_pages(q, self.k[layer], self.v[layer], table, items, scale, out=out, gate=gate, window=window, sink=sink, chunk=chunk, slopes=slopes,
                      out_scale=out_scale, pool=pool, pooled=self.pooled.get((layer, pool)))
        return out

    def _latent_ok(self, layer: int, q: torch.Tensor) -> bool:
        _, D, Dv = self.shapes[layer]
        bs = self.block_size
        return (self.values_in_keys[layer] and q.dtype == torch.bfloat16 and q.is_contiguous() and D <= 576 and Dv <= 512 and q.shape[0] < 65536
                and bs >= 8 and (128 % bs == 0 or bs % 128 == 0))

    def _latent_rows(self, layer: int, q: torch.Tensor, visible: torch.Tensor, slots: torch.Tensor | None, scale: float, out: torch.Tensor,
                     n_splits: int = 0) -> torch.Tensor:
        """Rows of queries in the latent space over latent rows (the tensor-core kernel)."""
        B, H, W = q.shape
        Dv = self.shapes[layer][2]
        if n_splits <= 0:
            n_splits = max(1, min(16, 148 // (B * ((H + 31) // 32))))
        lib = _native.kernels()
        n_scr = int(lib.ft_paged_decode_scratch(B, H, Dv, n_splits))
        scratch = F._get_scratch("paged_decode", n_scr, q.device) if n_scr else None
        rc = lib.ft_latent_decode(q.data_ptr(), self.k[layer].data_ptr(), self.block_table.data_ptr(), _ptr(slots), visible.data_ptr(), out.data_ptr(),
                                  _ptr(scratch), B, H, W, Dv, out.stride(0), self.block_size, self.max_blocks, self.num_blocks, float(scale), n_splits,
                                  F._dev(q), F._stream())
        _native.check(rc, "ft_latent_decode")
        return out

    def gather_contexts(self, layer: int, spans: torch.Tensor, longest: int, out: torch.Tensor, pad: int) -> None:
        """Rows 0 .. n - 1 of a layer's keys of sequence ``slot``, contiguous from row ``first`` of ``out``, for every ``(slot, first, n)``
        of ``spans``, and zero rows up to a multiple of ``pad`` (device only)."""
        rc = _native.kernels().ft_latent_gather(self.k[layer].data_ptr(), self.sync_table().data_ptr(), spans.data_ptr(), spans.shape[0], longest,
                                                out.data_ptr(), out.shape[1] * out.element_size(), pad, self.block_size, self.max_blocks, self.num_blocks,
                                                F._dev(out), F._stream())
        _native.check(rc, "ft_latent_gather")

    def gather(self, layer: int, seq: int, length: int):
        """Contiguous ``[length, Hkv, D]`` K and ``[length, Hkv, Dv]`` V of one sequence (debug / reference path;
        paged_attention.rs ``get_keys`` / ``get_values``)."""
        pages = self._pages[seq][: (length + self.block_size - 1) // self.block_size]
        idx = torch.tensor(pages, device=self.k[layer].device, dtype=torch.long)
        k = self.k[layer][idx].flatten(0, 1)[:length]
        v = self.v[layer][idx].flatten(0, 1)[:length]
        return k, v

    # ---- accessors under the reference's names (paged_attention.rs:359-395; there one object per
    # sequence, here one per model, hence the ``seq`` argument)
    def get_keys(self, seq: int, layer: int = 0) -> torch.Tensor:
        return self.gather(layer, seq, self.lengths[seq])[0]

    def get_values(self, seq: int, layer: int = 0) -> torch.Tensor:
        return self.gather(layer, seq, self.lengths[seq])[1]

    def len(self, seq: int | None = None) -> int:
        """Tokens of one sequence, or of all sequences together."""
        return self.lengths[seq] if seq is not None else sum(self.lengths)

    def is_empty(self, seq: int | None = None) -> bool:
        return self.len(seq) == 0

    def num_pages(self, seq: int | None = None) -> int:
        """Pages held by one sequence, or by all of them."""
        return len(self._pages[seq]) if seq is not None else self.pool.num_used

    def free_all(self) -> None:
        for s in range(self.max_seqs):
            if self._pages[s]:
                self.free_sequence(s)

    @staticmethod
    def _finish_reference(o, gate, out_scale):
        o = o if gate is None else ref.head_gate(o, gate)
        return o if out_scale == 1.0 else (o.float() * out_scale).to(o.dtype)

    def _decode_reference(self, layer, q, ctx_len, scale, seq_ids=None, window=None, sink=None, chunk=None, slopes=None, pool=None):
        """Host form of the paged-decode kernel, all rows at once: the pages of every row are gathered through
        the block table into a padded ``[B, L, Hkv, D]`` view and positions past a row's length are masked."""
        B, Hq, D = q.shape
        rows = torch.arange(B) if seq_ids is None else seq_ids.long().cpu()
        ctx = ctx_len.long().cpu()
        n_blk = int((int(ctx.max()) + self.block_size - 1) // self.block_size)
        pages = self._table_host[rows, :n_blk].long().clamp_(min=0)          # unreserved slots read page 0 and are masked
        Hkv, _, Dv = self.shapes[layer]
        k = self.k[layer][pages].reshape(B, n_blk * self.block_size, Hkv, D).float()
        v = self.v[layer][pages].reshape(B, n_blk * self.block_size, Hkv, Dv).float()
        qf = q.float().reshape(B, Hkv, Hq // Hkv, D)
        s = torch.einsum("bhgd,blhd->bhgl", qf, k) * scale
        at = torch.arange(n_blk * self.block_size)[None]
        dead = at >= ctx[:, None]
        if window:
            dead = dead | (at < ctx[:, None] - window)
        if chunk:
            dead = dead | (at < (ctx[:, None] - 1) // chunk * chunk)
        if slopes is not None:
            s = s - slopes.float().view(1, Hkv, Hq // Hkv, 1) * (ctx[:, None] - 1 - at).float()[:, None, None, :]
        s = s.masked_fill(dead[:, None, None, :], float("-inf"))
        seen = (ctx - window).clamp(min=0) // pool if pool else torch.zeros(1, dtype=torch.long)
        if int(seen.max()):
            b = torch.arange(int(seen.max()))[None]
            kp, vp = (t[self._pooled_places(rows[:, None], b, pool)].float() for t in self.pooled[layer, pool])
            sp = torch.einsum("bhgd,blhd->bhgl", qf, kp) * scale
            s = torch.cat([s, sp.masked_fill((b >= seen[:, None])[:, None, None, :], float("-inf"))], -1)
            v = torch.cat([v, vp], 1)
        if sink is not None:                              # one more column of the softmax, without a value
            s = torch.cat([s, sink.float().view(1, Hkv, Hq // Hkv, 1).expand(B, -1, -1, 1)], -1)
        o = torch.einsum("bhgl,blhd->bhgd", torch.softmax(s, -1)[..., :v.shape[1]], v)
        return o.reshape(B, Hq, Dv).to(q.dtype)


class PagedAttentionManager:
    """Multi-sequence front end: hands out sequence slots, grows and frees them
    (paged_attention.rs:447-532)."""

    def __init__(self, cache: PagedKVCache):
        self.cache = cache
        self._free_slots = list(range(cache.max_seqs - 1, -1, -1))
        self.active: dict[int, int] = {}
        self._filled: dict[int, dict[int, int]] = {}        # tokens written through append_kv, per sequence and layer

    def add_sequence(self, prompt_len: int = 0) -> int:
        if not self._free_slots:
            raise OutOfPages("no free sequence slot")
        s = self._free_slots.pop()
        try:
            self.cache.reserve(s, prompt_len)
        except OutOfPages:
            self.cache.free_sequence(s)
            self._free_slots.append(s)
            raise
        self.active[s] = prompt_len
        return s

    def extend(self, seq: int, n_tokens: int = 1) -> int:
        new_len = self.active[seq] + n_tokens
        self.cache.reserve(seq, new_len)
        self.active[seq] = new_len
        return new_len

    def remove_sequence(self, seq: int) -> None:
        self.cache.free_sequence(seq)
        del self.active[seq]
        self._filled.pop(seq, None)
        self._free_slots.append(seq)
        self._free_slots.sort(reverse=True)  # lowest free slot is handed out first

    @property
    def free_pages(self) -> int:
        return self.cache.pool.num_free

    def num_sequences(self) -> int:
        return len(self.active)

    def pool_utilization(self) -> float:
        """Fraction of the pages in use, 0.0 .. 1.0 (paged_attention.rs:525)."""
        pool = self.cache.pool
        return pool.num_used / pool.num_total if pool.num_total else 0.0

    def pool(self) -> PagePool:
        return self.cache.pool

    # ---- the reference's data-carrying calls (paged_attention.rs:485-510): its manager owns one
    # cache per sequence; here one paged cache serves every layer, hence the ``layer`` argument
    def append_kv(self, seq_id: int, key: torch.Tensor, value: torch.Tensor, layer: int = 0) -> None:
        """Append ``key`` / ``value`` (``[new_tokens, num_kv_heads, head_dim]``, or flat with that many
        elements) to sequence ``seq_id``.  Layer 0 grows the sequence (pages are taken from the pool as
        needed); other layers write the same positions, so append layer 0 first."""
        if seq_id not in self.active:
            raise ValueError("PagedAttentionManager: invalid sequence id %d" % seq_id)
        c = self.cache
        key, value = key.reshape(-1, c.n_kv_heads, c.head_dim), value.reshape(-1, c.n_kv_heads, c.head_dim)
        if key.shape != value.shape:
            raise ValueError("append_kv: key %s and value %s differ" % (tuple(key.shape), tuple(value.shape)))
        n = key.shape[0]
        filled = self._filled.setdefault(seq_id, {})
        start = filled.get(layer, 0)
        if start + n > self.active[seq_id]:
            self.extend(seq_id, start + n - self.active[seq_id])
        dev = c.k[layer].device
        pos = torch.arange(start, start + n, dtype=torch.int32, device=dev)
        sid = torch.full((n,), seq_id, dtype=torch.int32, device=dev)
        c.append(layer, key.to(device=dev, dtype=c.k[layer].dtype), value.to(device=dev, dtype=c.v[layer].dtype), pos, sid)
        filled[layer] = start + n

    def get_kv(self, seq_id: int, layer: int = 0):
        """``(keys, values)`` of a sequence as contiguous ``[tokens, num_kv_heads, head_dim]`` tensors."""
        if seq_id not in self.active:
            raise ValueError("PagedAttentionManager: invalid sequence id %d" % seq_id)
        return self.cache.gather(layer, seq_id, self._filled.get(seq_id, {}).get(layer, self.active[seq_id]))


class PagedSession:
    """A fixed set of equally long sequences on a paged cache of their own, for callers that think in ``[B, S]`` tensors
    (``models.generation``).  ``model`` offers ``make_paged_cache`` and ``paged_forward``."""

    def __init__(self, model, batch: int, max_len: int, block_size: int = 16):
        pages = batch * ((max_len + block_size - 1) // block_size)
        self.model, self.len = model, 0
        self.cache = model.make_paged_cache(pages, block_size, batch, max_len)
        self.manager = PagedAttentionManager(self.cache)
        self.slots = [self.manager.add_sequence(0) for _ in range(batch)]

    def extend(self, input_ids: torch.Tensor, last_token_only: bool = False) -> torch.Tensor:
        """Append ``input_ids [B, S]`` to the sequences; logits ``[B, S or 1, V]``."""
        B, S = input_ids.shape
        if B != len(self.slots):
            raise ValueError("PagedSession: %d sequences, got a batch of %d" % (len(self.slots), B))
        want = [S - 1] if last_token_only else list(range(S))
        entries = []
        for slot, tokens in zip(self.slots, input_ids.tolist()):
            self.manager.extend(slot, S)
            entries.append((slot, tokens, self.len, want))
        self.len += S
        logits = self.model.paged_forward(RaggedBatch(entries, self.cache.device), self.cache)
        return logits.view(B, len(want), -1)

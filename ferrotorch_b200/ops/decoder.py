"""Front ends of the kernels that decoders over paged caches use beside the projections and the attention: RMS
norm of fp32 residual rows, norm after a residual sum, norms of parts and powers of a row, the per-head pass between projection and
attention (``csrc/decoder_rows.cu``), residuals of several streams and n-gram embeddings (``csrc/streams.cu``), short convolution and gated linear recurrence
(``csrc/recurrent.cu``), matrix memories and state-space heads (``csrc/matrix_memory.cu``), the pass ahead of latent attention
(``csrc/latent_attn.cu``), routing and grouped products of expert layers and products by blocks (``csrc/grouped_gemm.cu``).

CUDA tensors run the kernels (bf16 on the tensor cores where there is a product, fp32 in true 32-bit); CPU tensors run
the plain forms of :mod:`ferrotorch_b200.ops.reference`."""
from __future__ import annotations

from dataclasses import dataclass
from typing import NamedTuple

import torch

from .. import _native
from . import functional as F
from . import reference as ref

_i, _ll, _f, _vp = _native._i, _native._ll, _native._f, _native._vp
_native.register_protos({
    "ft_rms_rows": (_i, [_vp, _vp, _i, _i] + [_vp] * 3 + [_i, _i, _vp, _vp] + [_i] * 4 + [_ll] * 4 + [_f, _f, _i, _vp]),
    "ft_qkv_head_finish": (_i, [_vp, _ll] + [_vp] * 8 + [_i] * 11 + [_f] + [_i] * 5 + [_vp]),
    "ft_sum_norm_rows": (_i, [_vp, _ll, _vp, _i, _i, _vp, _vp, _ll, _vp, _vp, _ll, _i, _vp, _vp, _i, _vp, _ll, _f] + [_vp] * 3 + [_ll, _vp, _ll] + [_i] * 5 + [_f, _i, _vp]),
    "ft_part_norm": (_i, [_vp, _ll, _vp] + [_i] * 5 + [_f, _i, _i, _vp]),
    "ft_poly_norm": (_i, [_vp, _ll, _vp, _ll, _vp] + [_i] * 3 + [_f, _i, _i, _vp]),
    "ft_causal_conv": (_i, [_vp, _ll] + [_vp] * 4 + [_ll] + [_vp] * 3 + [_i] * 7 + [_vp]),
    "ft_conv_tail": (_i, [_vp, _ll, _vp, _vp] + [_i] * 5 + [_vp]),
    "ft_rglru_gates": (_i, [_vp, _ll] + [_vp] * 4 + [_i] * 3 + [_vp, _vp, _i] + [_vp] * 4 + [_ll, _vp, _ll] + [_i] * 3 + [_vp]),
    "ft_rglru_scan": (_i, [_vp] * 3 + [_ll, _vp, _ll, _vp, _vp, _i, _vp, _ll, _vp] + [_i] * 4 + [_vp]),
    "ft_moe_max_items": (_i, [_i, _i]),
    "ft_moe_route": (_i, [_vp, _ll, _vp, _vp, _ll] + [_i] * 6 + [_vp, _vp, _i, _vp, _i] + [_vp] * 5 + [_i, _vp, _vp, _i, _vp]),
    "ft_block_linear": (_i, [_vp, _ll, _i, _vp] + [_i] * 6 + [_vp, _ll, _i, _vp, _ll] + [_i] * 3 + [_vp]),
    "ft_few_outputs": (_i, [_vp, _ll, _vp, _vp] + [_i] * 5 + [_vp]),
    "ft_stream_step": (_i, [_vp, _ll, _ll, _vp, _i] + [_vp] * 4 + [_i, _vp, _ll, _vp, _ll, _i, _vp, _vp, _i, _vp, _ll, _vp, _vp, _ll] + [_i] * 3 + [_f, _i, _i, _vp]),
    "ft_embed_bigram": (_i, [_vp] * 8 + [_ll, _i, _i, _ll, _ll, _f, _vp, _i] + [_vp] * 3 + [_i] * 3 + [_f] + [_i] * 5 + [_vp]),
    "ft_softcap": (_i, [_vp, _ll, _f, _i, _vp]),
    "ft_latent_finish": (_i, [_vp, _ll, _vp, _i] + [_vp] * 6 + [_i] * 11 + [_f] + [_i] * 5 + [_vp]),
    "ft_memory_scratch": (_ll, [_i] * 5),
    "ft_memory_chunks": (_i, [_vp] * 4 + [_ll, _vp, _ll, _i] + [_vp] * 7 + [_ll] + [_i] * 4 + [_f] * 4 + [_i, _vp, _i, _vp, _vp, _i, _vp, _i, _vp]),
    "ft_memory_steps": (_i, [_vp] * 4 + [_ll, _vp, _ll, _i] + [_vp] * 7 + [_ll] + [_i] * 4 + [_f] * 4 + [_vp] * 3 + [_i] * 3 + [_vp]),
    "ft_state_scratch": (_ll, [_i] * 5),
    "ft_state_chunks": (_i, [_vp] * 3 + [_ll, _vp, _ll, _vp, _ll] + [_vp] * 5 + [_ll] + [_i] * 5 + [_vp, _i, _vp, _vp, _i, _vp, _i, _vp]),
    "ft_state_steps": (_i, [_vp] * 3 + [_ll, _vp, _ll, _vp, _ll] + [_vp] * 5 + [_ll] + [_i] * 4 + [_vp] * 3 + [_i] * 3 + [_vp]),
    "ft_grouped_gemm": (_i, [_vp, _ll, _i] + [_vp] * 3 + [_i] * 5 + [_vp, _i, _vp, _ll] + [_i] * 4 + [_vp]),
})


def _ptr(t: torch.Tensor | None):
    return t.data_ptr() if t is not None else None


# --------------------------------------------------------------------------- RMS norm of residual rows
def rms_rows(x: torch.Tensor, weight: torch.Tensor, eps: float, *, count: int | None = None, offset: float = 0.0,
             rows: torch.Tensor | None = None, pending: tuple | None = None, update: bool = False,
             out_dtype: torch.dtype | None = None):
    """RMS norm of fp32 residual rows ``x [N, H]`` (padding beyond ``count`` elements is zero) times ``offset + weight``.

    ``rows``: normalise ``x[rows]``.  ``pending = (terms, where)``: row i first gains ``terms[where[i, j]]`` for all j
    (``where [N, n]`` int32); with ``update`` the sum is also stored back into ``x`` (not with ``rows``)."""
    dt, count = out_dtype or x.dtype, count or x.shape[1]
    if not x.is_cuda:
        if pending is not None:
            total = x + pending[0][pending[1].long()].float().sum(1)
            x = x.copy_(total) if update else total
        xs = x if rows is None else x[rows]
        return ref.rms_rows(xs, weight, eps, count, offset).to(dt)
    n = x.shape[0] if rows is None else rows.numel()
    y = torch.empty((n, x.shape[1]), device=x.device, dtype=dt)
    terms, where = pending[:2] if pending is not None else (None, None)
    rc = _native.kernels().ft_rms_rows(
        x.data_ptr(), _ptr(rows), x.shape[0], 0, x.data_ptr() if update else None, _ptr(terms), _ptr(where),
        where.shape[1] if where is not None else 0, terms.shape[0] if terms is not None else 0, weight.data_ptr(), y.data_ptr(),
        int(dt == torch.float32), n, x.shape[1], count, x.stride(0), x.stride(0), terms.stride(0) if terms is not None else 0,
        y.stride(0), float(eps), float(offset), F._dev(x), F._stream())
    _native.check(rc, "ft_rms_rows")
    return y


def embedding_rms(ids: torch.Tensor, table: torch.Tensor, weight: torch.Tensor, eps: float, *, count: int | None = None,
                  offset: float = 0.0, out_dtype: torch.dtype | None = None):
    """The gathered rows as the fp32 residual stream, and their RMS norm, from one kernel: ``(x, h)``."""
    dt, H = out_dtype or table.dtype, table.shape[1]
    if not table.is_cuda:
        x = table[ids].float()
        return x, ref.rms_rows(x, weight, eps, count or H, offset).to(dt)
    n = ids.numel()
    x = torch.empty((n, H), device=table.device, dtype=torch.float32)
    h = torch.empty((n, H), device=table.device, dtype=dt)
    rc = _native.kernels().ft_rms_rows(
        table.data_ptr(), ids.data_ptr(), table.shape[0], int(table.dtype == torch.bfloat16), x.data_ptr(), None, None, 0, 0,
        weight.data_ptr(), h.data_ptr(), int(dt == torch.float32), n, H, count or H, table.stride(0), H, 0, H, float(eps),
        float(offset), F._dev(table), F._stream())
    _native.check(rc, "ft_rms_rows")
    return x, h


# --------------------------------------------------------------------------- residuals of one or several streams
class SublayerTerms(NamedTuple):
    """What a sublayer adds to the residual, not yet summed: rows ``terms[where[i, j]]`` for all j (times ``weight[i, j]``), a dense
    row ``dense[i]`` (times ``dense_weight[i]``); where ``where[i, j]`` is negative, ``weight[i, j]`` times the sublayer's own input
    ``own[i]``."""
    terms: torch.Tensor | None = None
    where: torch.Tensor | None = None
    weight: torch.Tensor | None = None
    dense: torch.Tensor | None = None
    own: torch.Tensor | None = None
    dense_weight: torch.Tensor | None = None

    def total(self) -> torch.Tensor:
        """The sum, fp32."""
        y = self.dense.float() if self.dense is not None else 0.0
        if self.dense_weight is not None:
            y = y * self.dense_weight[:, None]
        if self.terms is None:
            return y
        t, w = self.terms[self.where.clamp(min=0).long()].float(), self.weight if self.weight is not None else torch.ones_like(self.where, dtype=torch.float32)
        if self.own is not None:
            t = torch.where(self.where[..., None] < 0, self.own.float()[:, None], t)
        return y + (t * w[..., None]).sum(1)


def sum_norm(x: torch.Tensor, y: SublayerTerms, gate: torch.Tensor | None, alpha: float, weight: torch.Tensor, eps: float, *, count: int,
             out_dtype: torch.dtype, ids: torch.Tensor | None = None, rows: torch.Tensor | None = None, last: torch.Tensor | None = None):
    """Norm after the sum: ``x' = norm(alpha x + sigmoid(gate) y) * weight`` (RMS over ``count`` elements), fp32 and as the next input.

    ``x [T, H]`` fp32 rows, or with ``ids`` rows ``x[ids]`` of an embedding table; ``gate [T, H]``: pre-activations, a view of a
    projection (``None``: no gate).  Returns ``(x', h)``; fp32 ``x`` is updated in place, and with an fp32 ``out_dtype`` both are one
    tensor.  ``rows``: only these rows, and no ``x'``; ``last``: weight of a second norm, of ``x'``, that ``h`` goes through."""
    H = x.shape[1]
    if not x.is_cuda:
        s = x[ids].float() if ids is not None else x
        t = y.total()
        s = alpha * s + (t if gate is None else t * torch.sigmoid(gate.float()))
        s = ref.rms_rows(s if rows is None else s[rows], weight, eps, count)
        h = s if last is None else ref.rms_rows(s, last, eps, count)
        return s, h.to(out_dtype)
    if y.own is not None:
        raise ValueError("sum_norm: terms of a sublayer's own input")
    T = x.shape[0] if ids is None else ids.numel()
    n = T if rows is None else rows.numel()
    new = None
    if rows is None:
        new = x if ids is None else torch.empty((T, H), device=x.device, dtype=torch.float32)
    same = new is not None and last is None and out_dtype == torch.float32
    h = None if same else torch.empty((n, H), device=x.device, dtype=out_dtype)
    t, dense = y.terms, y.dense
    rc = _native.kernels().ft_sum_norm_rows(
        x.data_ptr(), x.stride(0), _ptr(ids), x.shape[0], int(x.dtype == torch.bfloat16), _ptr(rows), _ptr(dense), dense.stride(0) if dense is not None else 0,
        _ptr(y.dense_weight), _ptr(t), t.stride(0) if t is not None else 0, t.shape[0] if t is not None else 0, _ptr(y.where), _ptr(y.weight),
        y.where.shape[1] if t is not None else 0, _ptr(gate), gate.stride(0) if gate is not None else 0, float(alpha), weight.data_ptr(), _ptr(last),
        _ptr(new), H, _ptr(h), H, int(out_dtype == torch.float32), n, T, H, count, float(eps), F._dev(x), F._stream())
    _native.check(rc, "ft_sum_norm_rows")
    return new, (new if same else h)


def stream_step(x: torch.Tensor, y: SublayerTerms, mix: torch.Tensor, out: torch.Tensor, into: torch.Tensor, weight: torch.Tensor, eps: float,
                *, count: int, out_dtype: torch.dtype, rows: torch.Tensor | None = None, update: bool = True):
    """All streams of the residual at once after a sublayer, and the next sublayer's input from them: ``(x', h)``.

    ``x [T, S, H]`` fp32 (a broadcast view when the streams are still equal): ``x'_t = sum_s mix[s, t] x_s + out[t] y``, in place
    where ``x`` is dense; ``h`` the RMS norm of ``sum_t into[t] x'_t`` times ``weight``.  ``rows``: only these rows; without
    ``update`` (always with ``rows``) the streams are not written."""
    T, S, H = x.shape
    if y.dense_weight is not None:
        raise ValueError("stream_step: dense rows have no weights of their own")
    if not x.is_cuda:
        new = torch.einsum("nsh,st->nth", x, mix) + out[:, None] * y.total()[:, None, :]
        u = torch.einsum("nth,t->nh", new if rows is None else new[rows], into)
        return new, ref.rms_rows(u, weight, eps, count).to(out_dtype)
    n = T if rows is None else rows.numel()
    update = update and rows is None
    dest = None
    if update:
        dest = x if x.is_contiguous() else torch.empty((T, S, H), device=x.device, dtype=torch.float32)
    h = torch.empty((n, H), device=x.device, dtype=out_dtype)
    t, own, dense = y.terms, y.own, y.dense
    rc = _native.kernels().ft_stream_step(
        x.data_ptr(), x.stride(0), x.stride(1) if S > 1 else 0, _ptr(rows), T, _ptr(dest), mix.data_ptr(), out.data_ptr(), into.data_ptr(), S, _ptr(dense),
        dense.stride(0) if dense is not None else 0, _ptr(t), t.stride(0) if t is not None else 0, t.shape[0] if t is not None else 0,
        _ptr(y.where), _ptr(y.weight), y.where.shape[1] if t is not None else 0, _ptr(own), own.stride(0) if own is not None else 0,
        weight.data_ptr(), h.data_ptr(), h.stride(0), n, H, count, float(eps), int(out_dtype == torch.float32), F._dev(x), F._stream())
    _native.check(rc, "ft_stream_step")
    return (dest if update else x), h


def embed_bigram(batch, cache, table: torch.Tensor, bigram: torch.Tensor, scale: float, mul_prev: int, mul_cur: int, into: torch.Tensor,
                 weight: torch.Tensor, eps: float, *, count: int, out_dtype: torch.dtype):
    """``x = scale * table[token] + bigram[row]`` of a ragged batch (fp32 ``[T, H]``) and the RMS norm of ``sum(into) x``: ``(x, h)``.

    ``row = (previous * mul_prev + token * mul_cur) mod buckets``, the last row of ``bigram [buckets + 1, H]`` for the first token of
    a sequence.  The cache keeps the tokens (:meth:`PagedKVCache.keep_tokens`): a portion finds its previous token there."""
    T, H, buckets = batch.n_rows, table.shape[1], bigram.shape[0] - 1
    pages = cache.token_pages
    cache.sync_table()
    if not table.is_cuda:
        pos, slots, bs = batch.positions.long(), batch.slots.long(), cache.block_size
        before = (pos - 1).clamp(min=0)
        held = pages[cache._table_host[slots, before // bs].long().clamp(min=0), before % bs].long()
        prev = torch.where(pos > batch.starts, torch.cat([batch.tokens[:1], batch.tokens[:-1]]), held)
        row = torch.where(pos > 0, (prev * mul_prev + batch.tokens * mul_cur) % buckets, buckets)
        pages[cache._table_host[slots, pos // bs].long(), pos % bs] = batch.tokens.int()
        x = scale * table[batch.tokens].float() + bigram[row].float()
        return x, ref.rms_rows(x * into.sum(), weight, eps, count).to(out_dtype)
    x = torch.empty((T, H), device=table.device, dtype=torch.float32)
    h = torch.empty((T, H), device=table.device, dtype=out_dtype)
    rc = _native.kernels().ft_embed_bigram(
        batch.tokens.data_ptr(), batch.positions.data_ptr(), batch.starts.data_ptr(), batch.slots.data_ptr(), cache.block_table.data_ptr(),
        pages.data_ptr(), table.data_ptr(), bigram.data_ptr(), table.stride(0), table.shape[0], buckets, mul_prev, mul_cur, float(scale),
        into.data_ptr(), into.numel(), weight.data_ptr(), x.data_ptr(), h.data_ptr(), T, H, count, float(eps), int(out_dtype == torch.float32),
        cache.block_size, cache.max_blocks, cache.num_blocks, F._dev(table), F._stream())
    _native.check(rc, "ft_embed_bigram")
    return x, h


def softcap_(z: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(z / cap)`` on contiguous fp32 logits, in place."""
    if not z.is_cuda:
        return z.copy_(cap * torch.tanh(z / cap))
    rc = _native.kernels().ft_softcap(z.data_ptr(), z.numel(), float(cap), F._dev(z), F._stream())
    _native.check(rc, "ft_softcap")
    return z


# --------------------------------------------------------------------------- norms inside sublayers
def part_norm_(y: torch.Tensor, weight: torch.Tensor, parts: int, eps: float, *, heads: int, vdim: int) -> torch.Tensor:
    """RMS norm of ``parts`` equal runs of every row on their own, times ``weight``, in place.  Rows ``[T, heads * vp]`` are heads of
    ``vdim`` elements padded to ``vp``, and runs count the true elements."""
    T, vp = y.shape[0], y.shape[1] // heads
    if not y.is_cuda:
        true = y.unflatten(1, (heads, vp))[:, :, :vdim]
        true.copy_(ref.part_rms(true.flatten(1), weight.view(heads, vp)[:, :vdim].flatten(), parts, eps).view(T, heads, vdim))
        return y
    rc = _native.kernels().ft_part_norm(y.data_ptr(), y.stride(0), weight.data_ptr(), T, heads, vdim, vp, parts, float(eps), int(y.dtype == torch.float32),
                                        F._dev(y), F._stream())
    _native.check(rc, "ft_part_norm")
    return y


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float, *, count: int) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e``, ``coef [4] = (a, b, c, e)`` fp32, N dividing a row (zero beyond ``count`` elements) by its
    root mean square."""
    if not z.is_cuda:
        return ref.poly_norm(z, coef, count, eps).to(z.dtype)
    out = torch.empty(z.shape, device=z.device, dtype=z.dtype)
    rc = _native.kernels().ft_poly_norm(z.data_ptr(), z.stride(0), out.data_ptr(), out.stride(0), coef.data_ptr(), z.shape[0], z.shape[1], count, float(eps),
                                        int(z.dtype == torch.float32), F._dev(z), F._stream())
    _native.check(rc, "ft_poly_norm")
    return out


# --------------------------------------------------------------------------- projection -> attention, per head
def qkv_head_finish(packed: torch.Tensor, cache, layer: int, batch, *, heads: int, dim: int, q_off: int = 0, k_off: int = 0,
                    v_off: int = 0, own_keys: bool = True, q_weight: torch.Tensor | None = None,
                    k_weight: torch.Tensor | None = None, true_dim: int | None = None, eps: float = 1e-5,
                    table: torch.Tensor | None = None) -> None:
    """Everything between a packed projection ``[T, N]`` and its attention, in one kernel: RMS norm of every query and key
    head (weights ``[dim]``, shared by the heads; ``None``: no norm), rotation of their leading elements by ``table``
    ``[positions, half, 2]`` (cos, sin), keys and values into the pages of ``layer``.  Queries change in place.
    ``own_keys`` false: the row has queries only, ``layer`` was filled by another layer of the model."""
    true_dim = true_dim or dim
    Hkv, D, Dv = cache.shapes[layer]
    if D != dim:
        raise ValueError("qkv_head_finish: query heads of %d over cached keys of %d" % (dim, D))
    cache.sync_table()
    if not packed.is_cuda:
        def finish(t, w):
            t = t.float() if w is None else ref.projection_rms(t, w, eps, true_dim)
            return t if table is None else ref.rotate_leading(t, table, batch.positions)

        q = packed[:, q_off:q_off + heads * dim]
        if own_keys:
            k = packed[:, k_off:k_off + Hkv * D].unflatten(1, (Hkv, D))
            v = packed[:, v_off:v_off + Hkv * Dv].unflatten(1, (Hkv, Dv))
            cache.append(layer, finish(k, k_weight), v, batch.positions, batch.slots)
        q.copy_(finish(q.unflatten(1, (heads, dim)), q_weight).flatten(1))
        return
    rc = _native.kernels().ft_qkv_head_finish(
        packed.data_ptr(), packed.stride(0), batch.positions.data_ptr(), batch.slots.data_ptr(), cache.block_table.data_ptr(),
        cache.k[layer].data_ptr() if own_keys else None, cache.v[layer].data_ptr() if own_keys else None, _ptr(q_weight),
        _ptr(k_weight), _ptr(table), packed.shape[0], q_off, heads, k_off, v_off, Hkv, dim, Dv, true_dim,
        table.shape[1] if table is not None else 0, table.shape[0] if table is not None else 0, float(eps),
        int(packed.dtype == torch.float32), cache.block_size, cache.max_blocks, cache.num_blocks, F._dev(packed), F._stream())
    _native.check(rc, "ft_qkv_head_finish")


def latent_finish(packed: torch.Tensor, cache, layer: int, batch, *, heads: int, q_off: int, q_head: int, q_rot: int, c_off: int, rank: int,
                  rank_pad: int, weight: torch.Tensor, eps: float, table: torch.Tensor, q_lat: torch.Tensor | None = None) -> None:
    """Everything between a packed projection and its latent attention, in one kernel: RMS norm of the latent (``rank`` of ``rank_pad``
    elements at ``c_off``, ``weight [rank_pad]``), rotation of the key part behind it and of the part at ``q_rot`` of every query
    head (heads of ``q_head`` elements from ``q_off``; pairs of neighbours, ``table [positions, half, 2]``), the row into its page
    (and nowhere else).  The queries change in place, except that the first rows' rotated parts go to ``q_lat [rows, heads,
    rank_pad + rot_pad]``, behind the place of their latent part."""
    width = cache.shapes[layer][1]
    rot_pad, half = width - rank_pad, table.shape[1]
    n_lat = q_lat.shape[0] if q_lat is not None else 0
    cache.sync_table()
    if not packed.is_cuda:
        row = packed[:, c_off:c_off + width].float()
        c = ref.rms_rows(row[:, :rank_pad], weight, eps, rank)
        row = torch.cat([c, ref.rotate_pairs(row[:, None, rank_pad:], table, batch.positions)[:, 0]], 1).to(packed.dtype)
        pos = batch.positions.long()
        cache.k[layer][cache._table_host[batch.slots.long(), pos // cache.block_size].long(), pos % cache.block_size, 0] = row
        q = packed[:, q_off:q_off + heads * q_head].unflatten(1, (heads, q_head))[:, :, q_rot:q_rot + rot_pad]
        turned = ref.rotate_pairs(q.float(), table, batch.positions).to(packed.dtype)
        if n_lat:
            q_lat[:, :, rank_pad:] = turned[:n_lat]
        q[n_lat:] = turned[n_lat:]
        return
    rc = _native.kernels().ft_latent_finish(
        packed.data_ptr(), packed.stride(0), _ptr(q_lat), n_lat, batch.positions.data_ptr(), batch.slots.data_ptr(), cache.block_table.data_ptr(),
        cache.k[layer].data_ptr(), weight.data_ptr(), table.data_ptr(), packed.shape[0], heads, q_off, q_head, q_rot, c_off, rank_pad, rank, rot_pad,
        half, table.shape[0], float(eps), int(packed.dtype == torch.float32), cache.block_size, cache.max_blocks, cache.num_blocks,
        F._dev(packed), F._stream())
    _native.check(rc, "ft_latent_finish")


def block_linear(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, a_col: int = 0, out_col: int = 0, gate: torch.Tensor | None = None,
                 glu: str | None = None, bn: int = 0) -> torch.Tensor:
    """Product by blocks of columns: block g of ``w [blocks, parts, N, K]`` takes columns ``g * a_col ..`` of ``a [T, ..]`` into columns
    ``g * out_col ..`` of ``out``.  One part: the product, times the sigmoid of ``gate`` (laid out like ``out``) when given; two
    parts with ``glu`` naming the activation: ``act(gate a) * (up a)``."""
    G, parts, N, K = w.shape
    T = a.shape[0]
    a_col, out_col = a_col or K, out_col or N
    if parts != (2 if glu else 1):
        raise ValueError("block_linear: %d parts with activation %r" % (parts, glu))
    if not a.is_cuda:
        for g in range(G):
            z = torch.einsum("tk,pnk->ptn", a[:, g * a_col:g * a_col + K].float(), w[g].float())
            z = z[0] if not glu else ref._ACTS[F._ACT_ID[glu]](z[0]) * z[1]
            if gate is not None:
                z = z * torch.sigmoid(gate[:, g * out_col:g * out_col + N].float())
            out[:, g * out_col:g * out_col + N] = z.to(out.dtype)
        return out
    rc = _native.kernels().ft_block_linear(
        a.data_ptr(), a.stride(0), T, w.data_ptr(), G, a_col, N, K, int(glu is not None), F._ACT_ID[glu] if glu else 0, out.data_ptr(),
        out.stride(0), out_col, _ptr(gate), gate.stride(0) if gate is not None else 0, int(a.dtype == torch.float32), bn, F._dev(a), F._stream())
    _native.check(rc, "ft_block_linear")
    return out


def few_outputs(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``h @ w.T`` with fp32 results for a few outputs: small batches on a kernel of their own, large ones as an ordinary product."""
    T, H = h.shape
    if not h.is_cuda or T > ROUTE_ROWS or w.shape[0] > 256:
        return F.linear_f32_out(h, w)
    z = torch.empty((T, w.shape[0]), device=h.device, dtype=torch.float32)
    rc = _native.kernels().ft_few_outputs(h.data_ptr(), h.stride(0), w.data_ptr(), z.data_ptr(), T, H, w.shape[0], int(h.dtype == torch.float32), F._dev(h),
                                          F._stream())
    _native.check(rc, "ft_few_outputs")
    return z


# --------------------------------------------------------------------------- recurrent blocks
def _span_list(batch) -> list:
    """``(slot, first row, first position, rows)`` of every entry of a batch, single tokens included (host path)."""
    slots, pos = batch.slots[:batch.n_single].tolist(), batch.positions[:batch.n_single].tolist()
    return [(s, i, p, 1) for i, (s, p) in enumerate(zip(slots, pos))] + [tuple(s) for s in batch.spans]


def causal_conv(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, state: torch.Tensor, batch, silu: bool = False) -> torch.Tensor:
    """Causal convolution per channel over the rows ``x [T, C]`` of a ragged batch: ``weight [taps, C]`` (the last one weighs
    the row itself), ``bias [C]``, fp32; ``silu``: of the result.  ``state [slots, taps - 1, C]`` holds the inputs ahead of a
    sequence's next row.  Rows that are a sequence's only token store theirs here, portions in :func:`conv_tail` or
    :func:`rglru_scan`."""
    taps, C = weight.shape
    u = torch.empty((x.shape[0], C), device=x.device, dtype=x.dtype)
    if not x.is_cuda:
        for slot, row, start, n in _span_list(batch):
            known = min(start, taps - 1)
            ahead = torch.cat([x.new_zeros(taps - 1 - known, C), state[slot, taps - 1 - known:]])
            z = torch.cat([ahead, x[row:row + n]]).float()
            out = sum(weight[j] * z[j:j + n] for j in range(taps)) + bias
            u[row:row + n] = ref.activation(out, "silu") if silu else out
            if row < batch.n_single:
                state[slot] = z[n:].to(state.dtype)
        return u
    rc = _native.kernels().ft_causal_conv(
        x.data_ptr(), x.stride(0), weight.data_ptr(), bias.data_ptr(), state.data_ptr(), u.data_ptr(), u.stride(0),
        batch.positions.data_ptr(), batch.slots.data_ptr(), batch.starts.data_ptr(), x.shape[0], batch.n_single, C, taps,
        int(silu), int(x.dtype == torch.float32), F._dev(x), F._stream())
    _native.check(rc, "ft_causal_conv")
    return u


def conv_tail(x: torch.Tensor, state: torch.Tensor, batch) -> None:
    """The last inputs of the portions of a batch, ``x [T, C]``, into the slots of a convolution's ``state [slots, taps - 1, C]``."""
    keep = state.shape[1]
    if not batch.spans or not keep:
        return
    if not x.is_cuda:
        for slot, row, _, n in batch.spans:
            state[slot] = torch.cat([state[slot], x[row:row + n].to(state.dtype)])[n:n + keep]
        return
    rc = _native.kernels().ft_conv_tail(x.data_ptr(), x.stride(0), state.data_ptr(), batch.span_table.data_ptr(), len(batch.spans), x.shape[1], keep,
                                        int(x.dtype == torch.float32), F._dev(x), F._stream())
    _native.check(rc, "ft_conv_tail")


def gated_recurrence(u: torch.Tensor, y: torch.Tensor, gates: torch.Tensor, r_bias: torch.Tensor, i_bias: torch.Tensor,
                     decay: torch.Tensor, state: torch.Tensor, batch, conv_x: torch.Tensor, conv_state: torch.Tensor,
                     out: torch.Tensor, bn: int = 0) -> torch.Tensor:
    """Real-gated linear recurrence over the rows of a ragged batch, times ``gelu(y)``, into ``out [T, C]``.

    ``u [T, C]``: the convolved branch; ``gates [blocks, 2, n, n]``: block-diagonal matrices of the recurrence and input
    gates with biases ``r_bias``, ``i_bias`` ``[C]``; ``decay [C]``: the logarithm of the decay at a full recurrence gate;
    ``state [slots, C]`` fp32.  ``conv_x``, ``conv_state``: the inputs and state of the convolution, whose last rows a
    portion leaves to the next.  Rows that are a sequence's only token take their step inside the product of the gates;
    portions are scanned."""
    blocks, _, n, _ = gates.shape
    T, C = u.shape
    if not u.is_cuda:
        z = torch.einsum("tbi,bpoi->ptbo", u.float().view(T, blocks, n), gates.float()).flatten(2)
        a, gain = ref.decay_and_gain(decay * torch.sigmoid(z[0] + r_bias))
        x = gain * torch.sigmoid(z[1] + i_bias) * u.float()
        keep = conv_state.shape[1]
        for slot, row, start, k in _span_list(batch):
            s = ref.linear_recurrence(a[row:row + k], x[row:row + k], state[slot] if start else torch.zeros_like(state[slot]))
            out[row:row + k] = (s * ref._ACTS[2](y[row:row + k].float())).to(out.dtype)
            state[slot] = s[-1]
            if row >= batch.n_single:
                conv_state[slot] = torch.cat([conv_state[slot], conv_x[row:row + k].to(conv_state.dtype)])[k:k + keep]
        return out
    a = torch.empty((T, C), device=u.device, dtype=torch.float32)
    x = torch.empty((T, C), device=u.device, dtype=torch.float32)
    f32, lib = int(u.dtype == torch.float32), _native.kernels()
    rc = lib.ft_rglru_gates(u.data_ptr(), u.stride(0), gates.data_ptr(), r_bias.data_ptr(), i_bias.data_ptr(), decay.data_ptr(), T,
                            blocks, n, a.data_ptr(), x.data_ptr(), batch.n_single, batch.positions.data_ptr(), batch.slots.data_ptr(),
                            state.data_ptr(), y.data_ptr(), y.stride(0), out.data_ptr(), out.stride(0), f32, bn, F._dev(u), F._stream())
    _native.check(rc, "ft_rglru_gates")
    rglru_scan(a, x, y, out, state, batch, conv_x, conv_state)
    return out


def rglru_scan(a: torch.Tensor, x: torch.Tensor, y: torch.Tensor, out: torch.Tensor, state: torch.Tensor, batch,
               conv_x: torch.Tensor, conv_state: torch.Tensor) -> None:
    """``S_t = a_t S_(t-1) + x_t`` over the portions of a batch (device only), ``out = S gelu(y)``; state and last inputs of the
    convolution go to the slots."""
    if not batch.spans:
        return
    rc = _native.kernels().ft_rglru_scan(
        a.data_ptr(), x.data_ptr(), y.data_ptr(), y.stride(0), out.data_ptr(), out.stride(0), state.data_ptr(),
        batch.span_table.data_ptr(), len(batch.spans), conv_x.data_ptr(), conv_x.stride(0), conv_state.data_ptr(),
        conv_state.shape[1], a.shape[1], int(y.dtype == torch.float32), F._dev(a), F._stream())
    _native.check(rc, "ft_rglru_scan")


MEMORY_CHUNK = 128       # tokens of a chunk of ft_memory_chunks
MEMORY_STEP_ROWS = 12    # a step whose portions have at most so many tokens runs them token by token


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, z: torch.Tensor, i_bias: torch.Tensor,
                  f_bias: torch.Tensor, norm: torch.Tensor, state, batch, out: torch.Tensor, *, heads: int, dim: int, vdim: int, cap: float,
                  eps: float, out_scale: float = 1.0, chunks: bool = False) -> torch.Tensor:
    """Matrix memories over the rows of a ragged batch: ``out = norm(o) * weight * sigmoid(gate) * out_scale`` per head (see
    ``csrc/matrix_memory.cu``).

    ``q, k [T, heads * dp]``, ``v, gate [T, heads * vp]``: parts of one packed projection (one row stride), heads padded from ``dim``
    and ``vdim``; ``z [T, 2 * n]`` fp32: pre-activations of the input gates and, from column n, of the forget gates; ``state``: what
    the sequences' slots hold (:class:`~ferrotorch_b200.nn.recurrent.MatrixMemoryState`).  Portions in bf16 run in chunks (short
    ones only with ``chunks``), everything else token by token."""
    T, n_gate = q.shape[0], z.shape[1] // 2
    if not q.is_cuda:
        qs, ks = (t.float().unflatten(1, (heads, -1)) for t in (q, k))
        vs = v.float().unflatten(1, (heads, -1))
        gi, gf = ref.memory_gates(z[:, :heads] + i_bias, z[:, n_gate:n_gate + heads] + f_bias, cap)
        for slot, row, start, n in _span_list(batch):
            if start == 0:
                for t in (state.S, state.n, state.m):
                    t[slot].zero_()
            r = slice(row, row + n)
            o = ref.matrix_memory(qs[r] * dim ** -0.5, ks[r], vs[r], gi[r], gf[r], state.S[slot], state.n[slot], state.m[slot])
            o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / vdim + eps)
            out[r] = (o.flatten(1) * norm * torch.sigmoid(gate[r].float()) * out_scale).to(out.dtype)
        return out
    dp, vp = state.S.shape[2:]
    lib, f32 = _native.kernels(), q.dtype == torch.float32
    args = (q.data_ptr(), k.data_ptr(), v.data_ptr(), gate.data_ptr(), q.stride(0), z.data_ptr(), z.stride(0), n_gate, i_bias.data_ptr(),
            f_bias.data_ptr(), norm.data_ptr(), state.S.data_ptr(), state.n.data_ptr(), state.m.data_ptr(), out.data_ptr(), out.stride(0), heads, dp, vp,
            vdim, dim ** -0.5, float(cap), float(eps), float(out_scale))

    def steps(spans, items):
        rc = lib.ft_memory_steps(*args, _ptr(spans), batch.positions.data_ptr(), batch.slots.data_ptr(), items, int(f32), F._dev(q), F._stream())
        _native.check(rc, "ft_memory_steps")

    if batch.n_single:
        steps(None, batch.n_single)
    if not batch.spans:
        return out
    if f32 or dp > 128 or vp > 256 or (batch.longest <= MEMORY_STEP_ROWS and not chunks):
        steps(batch.span_table, len(batch.spans))
        return out
    first, table = batch.chunk_table(MEMORY_CHUNK)
    scratch = F._get_scratch("matrix_memory", (int(lib.ft_memory_scratch(T, heads, dp, vp, table.shape[0])) + 3) // 4, q.device)
    rc = lib.ft_memory_chunks(*args, T, batch.span_table.data_ptr(), len(batch.spans), first.data_ptr(), table.data_ptr(), table.shape[0], scratch.data_ptr(),
                              F._dev(q), F._stream())
    _native.check(rc, "ft_memory_chunks")
    return out


def state_space(u: torch.Tensor, gate: torch.Tensor, step: torch.Tensor, step_bias: torch.Tensor, rate: torch.Tensor, skip: torch.Tensor, state: torch.Tensor,
                batch, out: torch.Tensor, *, heads: int, groups: int, chunks: bool = False) -> torch.Tensor:
    """State-space heads over the rows of a ragged batch (see ``csrc/matrix_memory.cu``): ``S <- exp(-rate dt) S + dt B x^T`` with ``dt =
    softplus(step + step_bias)``, ``out = (S^T C + skip x) silu(gate)``.

    ``u [T, heads * vp + 2 * groups * np]``: x of the heads, B and C of the groups (head h uses group ``h // (heads / groups)``), padded
    sizes; ``gate, out [T, heads * vp]``; ``step [T, >= heads]`` fp32; ``step_bias, rate, skip [heads]``; ``state [slots, heads, np, vp]``
    fp32.  Portions in bf16 run in chunks (short ones only with ``chunks``), everything else token by token."""
    np_, vp = state.shape[2:]
    hx, gn = heads * vp, groups * np_
    x, B, C = u[:, :hx], u[:, hx:hx + gn], u[:, hx + gn:]
    if not u.is_cuda:
        dt = torch.nn.functional.softplus(step[:, :heads] + step_bias, threshold=1e9)
        Bs, Cs = (t.float().unflatten(1, (groups, np_)).repeat_interleave(heads // groups, 1) for t in (B, C))
        xs = x.float().unflatten(1, (heads, vp))
        for slot, row, start, n in _span_list(batch):
            if start == 0:
                state[slot].zero_()
            r = slice(row, row + n)
            y = ref.state_space(Cs[r], Bs[r], xs[r], dt[r], rate, state[slot]) + skip[:, None] * xs[r]
            out[r] = (y.flatten(1) * ref.activation(gate[r].float(), "silu")).to(out.dtype)
        return out
    lib, f32, group, T = _native.kernels(), u.dtype == torch.float32, heads // groups, u.shape[0]
    args = (C.data_ptr(), B.data_ptr(), x.data_ptr(), u.stride(0), gate.data_ptr(), gate.stride(0), step.data_ptr(), step.stride(0), step_bias.data_ptr(),
            rate.data_ptr(), skip.data_ptr(), state.data_ptr(), out.data_ptr(), out.stride(0), heads, group, np_, vp)

    def steps(spans, items):
        rc = lib.ft_state_steps(*args, _ptr(spans), batch.positions.data_ptr(), batch.slots.data_ptr(), items, int(f32), F._dev(u), F._stream())
        _native.check(rc, "ft_state_steps")

    if batch.n_single:
        steps(None, batch.n_single)
    if not batch.spans:
        return out
    if f32 or np_ > 128 or vp > 256 or (batch.longest <= MEMORY_STEP_ROWS and not chunks):
        steps(batch.span_table, len(batch.spans))
        return out
    first, table = batch.chunk_table(MEMORY_CHUNK)
    scratch = F._get_scratch("matrix_memory", (int(lib.ft_state_scratch(T, heads, np_, vp, table.shape[0])) + 3) // 4, u.device)
    rc = lib.ft_state_chunks(*args, T, batch.span_table.data_ptr(), len(batch.spans), first.data_ptr(), table.data_ptr(), table.shape[0], scratch.data_ptr(),
                             F._dev(u), F._stream())
    _native.check(rc, "ft_state_chunks")
    return out


# --------------------------------------------------------------------------- expert layers
@dataclass
class Routing:
    """Rows sorted by expert: ``sorted [T * top, H]``, ``place [T, top]`` (where a row's copies lie; -1: a choice without
    matrices), ``scale [T * top]`` (their weights), ``items`` / ``n_items`` (segments, on the device); ``gate [T]``: the sigmoid of one more output of the router."""
    index: torch.Tensor
    weight: torch.Tensor
    place: torch.Tensor
    scale: torch.Tensor
    items: torch.Tensor
    n_items: torch.Tensor
    sorted: torch.Tensor
    gate: torch.Tensor | None = None


_SCORES = {"sigmoid": 0, "softmax": 1}
ROUTE_ROWS = 512      # up to so many rows the routing kernel computes the logits itself


def moe_route(h: torch.Tensor, router: torch.Tensor, experts: int, top: int, *, identity: int = 0, score: str = "sigmoid",
              correction: torch.Tensor | None = None, normalize: bool = False, bias: torch.Tensor | None = None, gate: bool = False) -> Routing:
    """The ``top`` choices of every row of ``h [T, H]`` by its logits ``router h`` (fp32), and the rows sorted by expert.

    ``score``: ``sigmoid`` (the largest logits, weighted by their sigmoid) or ``softmax`` over all logits (the largest scores after
    adding ``correction``, weighted by the score itself; ``normalize``: over the sum of the chosen ones).  The router's first
    ``experts`` outputs are experts, ``identity`` more have no matrices.  ``bias`` (fp32, one per output) joins the logits; with ``gate``
    the output behind these is no choice: its sigmoid is returned.  ``router [>= experts + identity + gate, H]`` (padded rows are
    ignored)."""
    T, H = h.shape
    outputs = experts + identity
    if not h.is_cuda:
        z = h.float() @ router[:outputs].float().t()
        index, weight = ref.top_experts(z if bias is None else z + bias, top, score, correction, normalize)
        own = torch.sigmoid(h.float() @ router[outputs].float()) if gate else None
        order = index.flatten().argsort(stable=True)
        place = torch.empty_like(order)
        place[order] = torch.arange(order.numel())
        place[index.flatten() >= experts] = -1
        real = int((index < experts).sum())
        return Routing(index, weight, place.view(T, top).int(), weight.flatten()[order], index.flatten()[order][:real], torch.tensor(real),
                       h[order // top], own)
    lib, dev = _native.kernels(), h.device
    cap = int(lib.ft_moe_max_items(T * top, experts))
    ints = torch.empty(2 * T * top + 3 * cap + 1, device=dev, dtype=torch.int32)
    index, place, rest = ints[:T * top].view(T, top), ints[T * top:2 * T * top].view(T, top), ints[2 * T * top:]
    items, n_items = rest[:3 * cap].view(cap, 3), rest[3 * cap:]
    weight, scale = torch.empty((2, T * top), device=dev, dtype=torch.float32)
    rows = torch.empty((T * top, H), device=dev, dtype=h.dtype)
    own = torch.empty(T, device=dev, dtype=torch.float32) if gate else None
    logits = F.linear_f32_out(h, router) if T > ROUTE_ROWS else None
    rc = lib.ft_moe_route(h.data_ptr(), h.stride(0), router.data_ptr(), _ptr(logits), logits.stride(0) if logits is not None else 0, T, H,
                          experts, outputs, top, _SCORES[score], _ptr(correction), _ptr(bias), int(normalize), _ptr(own), int(h.dtype == torch.float32), index.data_ptr(), weight.data_ptr(), place.data_ptr(),
                          scale.data_ptr(), items.data_ptr(), cap, n_items.data_ptr(), rows.data_ptr(), F._dev(h), F._stream())
    _native.check(rc, "ft_moe_route")
    return Routing(index, weight.view(T, top), place, scale, items, n_items, rows, own)


def grouped_linear(a: torch.Tensor, w: torch.Tensor, routing: Routing, *, glu: str | None = None, seg_rows: int = 0,
                   bn: int = 0, scaled: bool = True, activation: str | None = None) -> torch.Tensor:
    """Rows sorted by expert through their expert's matrix: ``a [R, K]``, ``w [experts, parts, N, K]`` -> ``[R, N]``.  One part: the
    product, of which ``activation`` (relu2) is taken when named.  Two parts (gate, up) with ``glu`` naming the activation: ``act(gate r a) * (up r a)`` with r the row's routing
    weight (``scaled`` false: 1).  ``seg_rows``: an upper bound of the rows of one expert."""
    E, parts, N, K = w.shape
    R = a.shape[0]
    if parts != (2 if glu else 1) or activation not in (None, "relu2") or (glu and activation):
        raise ValueError("grouped_linear: %d parts with activation %r" % (parts, glu or activation))
    out = torch.empty((R, N), device=a.device, dtype=a.dtype)
    if not a.is_cuda:
        for e in routing.items.unique().tolist():
            rows = (routing.items == e).nonzero().flatten()
            z = torch.einsum("rk,pnk->prn", a[rows].float(), w[e].float())
            if glu:
                s = routing.scale[rows][:, None] if scaled else 1.0
                out[rows] = (ref._ACTS[F._ACT_ID[glu]](s * z[0]) * (s * z[1])).to(out.dtype)
            else:
                out[rows] = (ref.activation(z[0], activation) if activation else z[0]).to(out.dtype)
        return out
    rc = _native.kernels().ft_grouped_gemm(
        a.data_ptr(), a.stride(0), R, w.data_ptr(), routing.items.data_ptr(), routing.n_items.data_ptr(), routing.items.shape[0], E, N, K,
        int(glu is not None), routing.scale.data_ptr() if glu and scaled else None, F._ACT_ID[glu] if glu else (3 if activation else 0), out.data_ptr(), out.stride(0),
        seg_rows, int(a.dtype == torch.float32), bn, F._dev(a), F._stream())
    _native.check(rc, "ft_grouped_gemm")
    return out

"""Front ends of the kernels that pre-norm decoders over paged caches use beside the projections and the attention: RMS
norm of fp32 residual rows, the per-head pass between projection and attention (``csrc/decoder_rows.cu``), short
convolution and gated linear recurrence (``csrc/recurrent.cu``), routing and grouped products of expert layers
(``csrc/grouped_gemm.cu``).

CUDA tensors run the kernels (bf16 on the tensor cores where there is a product, fp32 in true 32-bit); CPU tensors run
the plain forms of :mod:`ferrotorch_b200.ops.reference`."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import _native
from . import functional as F
from . import reference as ref

_i, _ll, _f, _vp = _native._i, _native._ll, _native._f, _native._vp
_native.register_protos({
    "ft_rms_rows": (_i, [_vp, _vp, _i, _i] + [_vp] * 3 + [_i, _i, _vp, _vp] + [_i] * 4 + [_ll] * 4 + [_f, _f, _i, _vp]),
    "ft_qkv_head_finish": (_i, [_vp, _ll] + [_vp] * 8 + [_i] * 11 + [_f] + [_i] * 5 + [_vp]),
    "ft_causal_conv": (_i, [_vp, _ll] + [_vp] * 4 + [_ll] + [_vp] * 3 + [_i] * 6 + [_vp]),
    "ft_rglru_gates": (_i, [_vp, _ll] + [_vp] * 4 + [_i] * 3 + [_vp, _vp, _i] + [_vp] * 4 + [_ll, _vp, _ll] + [_i] * 3 + [_vp]),
    "ft_rglru_scan": (_i, [_vp] * 3 + [_ll, _vp, _ll, _vp, _vp, _i, _vp, _ll, _vp] + [_i] * 4 + [_vp]),
    "ft_moe_max_items": (_i, [_i, _i]),
    "ft_moe_route": (_i, [_vp, _ll, _vp, _vp, _ll] + [_i] * 5 + [_vp] * 5 + [_i, _vp, _vp, _i, _vp]),
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
    terms, where = pending if pending is not None else (None, None)
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


# --------------------------------------------------------------------------- recurrent blocks
def _span_list(batch) -> list:
    """``(slot, first row, first position, rows)`` of every entry of a batch, single tokens included (host path)."""
    slots, pos = batch.slots[:batch.n_single].tolist(), batch.positions[:batch.n_single].tolist()
    return [(s, i, p, 1) for i, (s, p) in enumerate(zip(slots, pos))] + [tuple(s) for s in batch.spans]


def causal_conv(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, state: torch.Tensor, batch) -> torch.Tensor:
    """Causal convolution per channel over the rows ``x [T, C]`` of a ragged batch: ``weight [taps, C]`` (the last one weighs
    the row itself), ``bias [C]``, fp32.  ``state [slots, taps - 1, C]`` holds the inputs ahead of a sequence's next row.
    Rows that are a sequence's only token store theirs here, portions in :func:`rglru_scan`."""
    taps, C = weight.shape
    u = torch.empty((x.shape[0], C), device=x.device, dtype=x.dtype)
    if not x.is_cuda:
        for slot, row, start, n in _span_list(batch):
            known = min(start, taps - 1)
            ahead = torch.cat([x.new_zeros(taps - 1 - known, C), state[slot, taps - 1 - known:]])
            z = torch.cat([ahead, x[row:row + n]]).float()
            u[row:row + n] = sum(weight[j] * z[j:j + n] for j in range(taps)) + bias
            if row < batch.n_single:
                state[slot] = z[n:].to(state.dtype)
        return u
    rc = _native.kernels().ft_causal_conv(
        x.data_ptr(), x.stride(0), weight.data_ptr(), bias.data_ptr(), state.data_ptr(), u.data_ptr(), u.stride(0),
        batch.positions.data_ptr(), batch.slots.data_ptr(), batch.starts.data_ptr(), x.shape[0], batch.n_single, C, taps,
        int(x.dtype == torch.float32), F._dev(x), F._stream())
    _native.check(rc, "ft_causal_conv")
    return u


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


# --------------------------------------------------------------------------- expert layers
@dataclass
class Routing:
    """Rows sorted by expert: ``sorted [T * top, H]``, ``place [T, top]`` (where a row's copies lie), ``scale [T * top]``
    (their weights), ``items`` / ``n_items`` (segments, on the device)."""
    index: torch.Tensor
    weight: torch.Tensor
    place: torch.Tensor
    scale: torch.Tensor
    items: torch.Tensor
    n_items: torch.Tensor
    sorted: torch.Tensor


ROUTE_ROWS = 512      # up to so many rows the routing kernel computes the logits itself


def moe_route(h: torch.Tensor, router: torch.Tensor, experts: int, top: int) -> Routing:
    """The ``top`` experts of every row of ``h [T, H]`` with the largest logits ``router h`` (fp32), weighted by the sigmoid of
    the logit, and the rows sorted by expert.  ``router [>= experts, H]`` (padded rows are ignored)."""
    T, H = h.shape
    if not h.is_cuda:
        index, weight = ref.top_experts(h.float() @ router[:experts].float().t(), top)
        order = index.flatten().argsort(stable=True)
        place = torch.empty_like(order)
        place[order] = torch.arange(order.numel())
        return Routing(index, weight, place.view(T, top).int(), weight.flatten()[order], index.flatten()[order], torch.tensor(T * top),
                       h[order // top])
    lib, dev = _native.kernels(), h.device
    cap = int(lib.ft_moe_max_items(T * top, experts))
    ints = torch.empty(2 * T * top + 3 * cap + 1, device=dev, dtype=torch.int32)
    index, place, rest = ints[:T * top].view(T, top), ints[T * top:2 * T * top].view(T, top), ints[2 * T * top:]
    items, n_items = rest[:3 * cap].view(cap, 3), rest[3 * cap:]
    weight, scale = torch.empty((2, T * top), device=dev, dtype=torch.float32)
    rows = torch.empty((T * top, H), device=dev, dtype=h.dtype)
    logits = F.linear_f32_out(h, router) if T > ROUTE_ROWS else None
    rc = lib.ft_moe_route(h.data_ptr(), h.stride(0), router.data_ptr(), _ptr(logits), logits.stride(0) if logits is not None else 0, T, H,
                          experts, top, int(h.dtype == torch.float32), index.data_ptr(), weight.data_ptr(), place.data_ptr(),
                          scale.data_ptr(), items.data_ptr(), cap, n_items.data_ptr(), rows.data_ptr(), F._dev(h), F._stream())
    _native.check(rc, "ft_moe_route")
    return Routing(index, weight.view(T, top), place, scale, items, n_items, rows)


def grouped_linear(a: torch.Tensor, w: torch.Tensor, routing: Routing, *, glu: str | None = None, seg_rows: int = 0,
                   bn: int = 0) -> torch.Tensor:
    """Rows sorted by expert through their expert's matrix: ``a [R, K]``, ``w [experts, parts, N, K]`` -> ``[R, N]``.  One part: the
    product.  Two parts (gate, up) with ``glu`` naming the activation: ``act(gate r a) * (up r a)`` with r the row's routing
    weight.  ``seg_rows``: an upper bound of the rows of one expert."""
    E, parts, N, K = w.shape
    R = a.shape[0]
    if parts != (2 if glu else 1):
        raise ValueError("grouped_linear: %d parts with activation %r" % (parts, glu))
    out = torch.empty((R, N), device=a.device, dtype=a.dtype)
    if not a.is_cuda:
        for e in routing.items.unique().tolist():
            rows = routing.items == e
            z = torch.einsum("rk,pnk->prn", a[rows].float(), w[e].float())
            if glu:
                s = routing.scale[rows][:, None]
                out[rows] = (ref._ACTS[F._ACT_ID[glu]](s * z[0]) * (s * z[1])).to(out.dtype)
            else:
                out[rows] = z[0].to(out.dtype)
        return out
    rc = _native.kernels().ft_grouped_gemm(
        a.data_ptr(), a.stride(0), R, w.data_ptr(), routing.items.data_ptr(), routing.n_items.data_ptr(), routing.items.shape[0], E, N, K,
        int(glu is not None), routing.scale.data_ptr() if glu else None, F._ACT_ID[glu] if glu else 0, out.data_ptr(), out.stride(0),
        seg_rows, int(a.dtype == torch.float32), bn, F._dev(a), F._stream())
    _native.check(rc, "ft_grouped_gemm")
    return out

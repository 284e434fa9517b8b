"""Parts of decoders over a paged cache: RMS norm of the fp32 residual stream, and attention with per-head query / key norm,
rotation, window, pooled blocks ahead of it, sink and an output gate per element, whose keys and values may be another layer's.

Sizes are padded at load time with zero weights like those of :mod:`~ferrotorch_b200.nn.packed_block`."""
from __future__ import annotations

import torch
from torch import nn

from ..ops import decoder as D
from ..ops import functional as F
from .packed_block import AttentionSpec, pad_heads, pad_to, round_up


def checked(owner: str, name: str, t: torch.Tensor | None, shape: tuple) -> torch.Tensor:
    if t is None or tuple(t.shape) != tuple(shape):
        raise ValueError("%s: %s must have shape %s, got %s" % (owner, name, tuple(shape), None if t is None else tuple(t.shape)))
    return t


def unpad_heads(t: torch.Tensor, heads: int, d: int) -> torch.Tensor:
    """The inverse of :func:`~ferrotorch_b200.nn.packed_block.pad_heads`."""
    return t.unflatten(0, (heads, -1))[:, :d].flatten(0, 1)


class ResidualRMSNorm(nn.Module):
    """``x / sqrt(mean(x^2) + eps) * (offset + w)`` on fp32 residual rows (``offset`` 1: the weight is stored around zero).
    The weight stays fp32 whatever the model's type."""

    def __init__(self, hidden_size: int, eps: float, offset: float = 0.0):
        super().__init__()
        self.hidden_size, self.eps, self.offset = hidden_size, eps, offset
        self.register_buffer("weight", torch.full((round_up(hidden_size, 8),), 0.0))
        self.weight[:hidden_size] = 1.0 - offset

    def load(self, weight: torch.Tensor) -> None:
        self.weight.copy_(pad_to(checked("ResidualRMSNorm", "weight", weight, (self.hidden_size,)).float(), self.weight.numel()))

    def unpack(self) -> torch.Tensor:
        return self.weight[:self.hidden_size]

    def forward(self, x: torch.Tensor, **kw) -> torch.Tensor:
        """Arguments of :func:`~ferrotorch_b200.ops.decoder.rms_rows`."""
        return D.rms_rows(x, self.weight, self.eps, count=self.hidden_size, offset=self.offset, **kw)

    def gather(self, ids: torch.Tensor, table: torch.Tensor, out_dtype: torch.dtype):
        return D.embedding_rms(ids, table, self.weight, self.eps, count=self.hidden_size, offset=self.offset, out_dtype=out_dtype)


class GatedAttention(nn.Module):
    """``W_o (attention(h) * sigmoid(W_g h))`` over a paged cache: added to the residual (:meth:`forward`) or left to the kernel that
    does (:meth:`terms`).

    One packed product ``[q | k | v | g | r]`` (``[q | g | r]`` when the keys are another layer's), one pass for norms, rotation and
    cache, the attention with sink, window, pooled blocks and gate, and the output product.  ``qk_norm``: RMS norm per head, by
    ``norm_weights`` with weights shared by the heads (a norm without weights and a rotation may change places); ``bias``: of queries,
    keys and values; ``sink``: one learned number per head in the denominator; ``gate``: per element; ``residual_gate``: pre-activations
    of a gate of the whole sublayer, ``rg`` with its bias ``rg.b``, ride along in the packed product."""

    def __init__(self, hidden_size: int, attn: AttentionSpec, eps: float, qk_norm: bool = True, sink: bool = True, gate: bool = True,
                 norm_weights: bool = True, bias: bool = False, residual_gate: bool = False):
        super().__init__()
        if attn.chunk is not None or attn.distance_bias or (attn.rotary is not None and attn.rotary.interleaved):
            raise ValueError("GatedAttention: no chunks, distance bias or rotation of neighbours")
        self.attn, self.eps, self.hidden_size, self.qk_norm, self.gated = attn, eps, hidden_size, qk_norm, gate
        self.norm_weights, self.bias, self.residual_gate = qk_norm and norm_weights, bias, residual_gate
        a, width = attn, round_up(hidden_size, 8)
        own = a.kv_from is None
        self.value_width = a.heads * a.padded_vdim
        sizes = (a.heads * a.padded_dim, a.kv_heads * a.padded_dim if own else 0, a.kv_heads * a.padded_vdim if own else 0,
                 self.value_width if gate else 0)
        at, self.segments = 0, []
        for n in sizes:
            self.segments.append((at, n))
            at += n
        self.gate_at = at
        at += width if residual_gate else 0
        self.register_buffer("in_proj", torch.zeros(at, width))
        self.register_buffer("in_bias", torch.zeros(at) if bias or residual_gate else None)
        self.register_buffer("out_proj", torch.zeros(width, self.value_width))
        ones = torch.ones(a.padded_dim)
        self.register_buffer("q_norm", (torch.zeros(a.padded_dim) if self.norm_weights else ones) if qk_norm else None)
        self.register_buffer("k_norm", (torch.zeros(a.padded_dim) if self.norm_weights else ones.clone()) if qk_norm and own else None)
        self.register_buffer("sink", torch.zeros(a.heads) if sink else None)

    def _parts(self) -> list:
        """``(name, first row of the packed product, heads, head size, padded head size, biased)`` of what it holds."""
        a, at = self.attn, [off for off, _ in self.segments]
        out = [("q", at[0], a.heads, a.dim, a.padded_dim, self.bias)]
        if a.kv_from is None:
            out += [("k", at[1], a.kv_heads, a.dim, a.padded_dim, self.bias), ("v", at[2], a.kv_heads, a.vdim, a.padded_vdim, self.bias)]
        if self.gated:
            out.append(("g", at[3], a.heads, a.vdim, a.padded_vdim, False))
        if self.residual_gate:
            out.append(("rg", self.gate_at, 1, self.hidden_size, self.in_proj.shape[1], True))
        return out

    def _shapes(self) -> dict:
        """True shapes of the weights by name."""
        a, W = self.attn, self.hidden_size
        out = {"o": (W, a.heads * a.vdim)}
        for name, _, heads, d, _, biased in self._parts():
            out[name] = (heads * d, W)
            if biased:
                out[name + ".b"] = (heads * d,)
        if self.norm_weights:
            out["q.norm"] = (a.dim,)
            if a.kv_from is None:
                out["k.norm"] = (a.dim,)
        if self.sink is not None:
            out["sink"] = (a.heads,)
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        """Weights by name (:meth:`tensor_names`), matrices ``[out, in]`` of the true sizes."""
        a = self.attn
        for name, shape in self._shapes().items():
            checked("GatedAttention", name, sd.get(name), shape)
        width = self.in_proj.shape[1]
        for name, at, heads, _, padded, biased in self._parts():
            n = heads * padded
            self.in_proj[at:at + n].copy_(pad_to(pad_heads(sd[name], heads, padded), n, width))
            if biased:
                self.in_bias[at:at + n].copy_(pad_heads(sd[name + ".b"].float(), heads, padded))
        self.out_proj.copy_(pad_to(pad_heads(sd["o"].t(), a.heads, a.padded_vdim).t(), width, self.value_width))
        if self.norm_weights:
            for buf, name in ((self.q_norm, "q.norm"), (self.k_norm, "k.norm")):
                if buf is not None:
                    buf.copy_(pad_to(sd[name].float(), a.padded_dim))
        if self.sink is not None:
            self.sink.copy_(sd["sink"].float())

    def unpack(self) -> dict:
        a, W = self.attn, self.hidden_size
        out = {}
        for name, at, heads, d, padded, biased in self._parts():
            out[name] = unpad_heads(self.in_proj[at:at + heads * padded, :W], heads, d)
            if biased:
                out[name + ".b"] = unpad_heads(self.in_bias[at:at + heads * padded], heads, d)
        out["o"] = unpad_heads(self.out_proj[:W].t(), a.heads, a.vdim).t()
        for buf, name, n in ((self.q_norm if self.norm_weights else None, "q.norm", a.dim), (self.k_norm if self.norm_weights else None, "k.norm", a.dim),
                             (self.sink, "sink", a.heads)):
            if buf is not None:
                out[name] = buf[:n]
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        dev = self.in_proj.device
        self.load({n: torch.ones(s, device=dev) if n.endswith("norm") else torch.randn(s, device=dev, generator=generator) * std
                   for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; biases, norm weights and sinks stay fp32."""
        self.in_proj, self.out_proj = self.in_proj.to(dtype), self.out_proj.to(dtype)

    def attend(self, h: torch.Tensor, batch, cache, layer: int) -> tuple:
        """The heads' results ``[T, heads * padded_vdim]`` for input ``h`` and the packed product; ``layer``: the (or its source's)
        place in the cache."""
        a = self.attn
        (qo, qn), (ko, _), (vo, _), (go, gn) = self.segments
        packed = F.linear_rows(h, self.in_proj, self.in_bias)
        D.qkv_head_finish(packed, cache, layer, batch, heads=a.heads, dim=a.padded_dim, q_off=qo, k_off=ko, v_off=vo,
                          own_keys=a.kv_from is None, q_weight=self.q_norm, k_weight=self.k_norm, true_dim=a.dim, eps=self.eps,
                          table=cache.rotary_table(a.rotary) if a.rotary is not None else None)
        if a.kv_from is None:
            cache.pool_blocks(layer, batch)
        heads = torch.empty((h.shape[0], a.heads, a.padded_vdim), device=h.device, dtype=h.dtype)
        gate = packed[:, go:go + gn].unflatten(1, (a.heads, a.padded_vdim)) if self.gated else None
        cache.attend(layer, packed[:, qo:qo + qn].unflatten(1, (a.heads, a.padded_dim)), batch, a.scale, gate=gate, out=heads,
                     window=a.window, sink=self.sink, pool=a.pool)
        return heads.flatten(1), packed

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch, cache, layer: int) -> None:
        """Adds the sublayer of input ``h`` to the fp32 residual ``x``."""
        F.residual_linear_(x, self.attend(h, batch, cache, layer)[0], self.out_proj)

    def terms(self, h: torch.Tensor, batch, cache, layer: int) -> tuple:
        """The sublayer's output and the pre-activations of its residual gate (a view; ``None`` without one)."""
        heads, packed = self.attend(h, batch, cache, layer)
        return D.SublayerTerms(dense=F.linear_rows(heads, self.out_proj)), packed[:, self.gate_at:] if self.residual_gate else None

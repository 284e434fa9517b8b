"""Inference blocks of decoders whose sublayers share one input: packed projections over a paged KV cache.

A layer whose attention and feed-forward read the same normalised input ``h`` and whose outputs are summed needs two
matrix products: one input projection ``[q | k | v | up | gate]`` and one output projection over the concatenation
``[attention heads | act(up)]``, which the GEMM adds onto the fp32 residual stream.  Between them run one row kernel
(:func:`~ferrotorch_b200.ops.functional.qkv_finish`) and the attention over the cache.

Sizes are padded at load time to what the kernels move (head sizes to multiples of 16, segments and the width to
multiples of 8) with zero weights, so every padded element of every activation is exactly zero and any size runs.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import functional as F
from ..ops import reference as ref


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def pad_to(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` in the leading corner of a zero tensor of ``shape``."""
    if tuple(t.shape) == shape:
        return t
    out = t.new_zeros(shape)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def pad_heads(t: torch.Tensor, heads: int, padded: int) -> torch.Tensor:
    """Rows (or elements) ``[heads * d, ...]`` with every head's ``d`` padded to ``padded``."""
    d = t.shape[0] // heads
    return pad_to(t.reshape(heads, d, *t.shape[1:]), heads, padded, *t.shape[1:]).flatten(0, 1)


@dataclass(frozen=True)
class YarnScaling:
    """Interpolation of slow rotary dimensions for contexts ``factor`` times as long as ``original``: dimensions that turn
    more than ``fast`` times over it keep their frequency, less than ``slow`` times have it divided, a linear ramp between."""
    factor: float
    original: float
    fast: float = 32.0
    slow: float = 1.0


@dataclass(frozen=True)
class WavelengthScaling:
    """Interpolation by wavelength for contexts ``factor`` times as long as ``original`` (Llama 3.1): dimensions that turn more than
    ``high`` times over it keep their frequency, less than ``low`` times have it divided, a linear transition between."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` elements of a head, frequencies ``base ** (-2 i / dims)``; pairs ``(i, i + dims / 2)``, or
    neighbours ``(2 i, 2 i + 1)`` when ``interleaved``."""
    dims: int
    base: float
    scaling: YarnScaling | WavelengthScaling | None = None
    interleaved: bool = False

    def table(self, positions: int, device="cpu") -> torch.Tensor:
        """cos and sin of every position, ``[positions, dims / 2, 2]`` fp32 (angles are computed in 64-bit)."""
        sc = self.scaling
        if isinstance(sc, WavelengthScaling):
            kind = {"type": "llama3", "factor": sc.factor, "original_max": sc.original, "low_freq_factor": sc.low, "high_freq_factor": sc.high}
        else:
            kind = None if sc is None else {"type": "yarn", "factor": sc.factor, "original_max": sc.original, "beta_fast": sc.fast,
                                            "beta_slow": sc.slow, "full_range": True, "mscale": "always"}
        return torch.stack(ref.rope_tables(self.dims, positions, self.base, kind), -1).contiguous().to(device)


def head_slopes(heads: int) -> torch.Tensor:
    """Slopes of a distance bias: ``2 ** (-8 (h + 1) / heads)`` for head h, fp32."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64).float()


@dataclass
class AttentionSpec:
    """One attention sublayer: ``heads`` query heads over ``kv_heads`` key/value heads of sizes ``dim`` / ``vdim``,
    ``score = (q . k) * scale``; ``temp_coef`` / ``temp_every``: query temperature (coef 0: none); ``window``: a query sees
    its last so many positions, its own included (``None``: all); ``chunk``: it sees those of its own chunk of so many positions,
    chunks counted from position 0 (``None``: all); ``distance_bias``: the distance of a key times the head's slope (:func:`head_slopes`)
    is taken off its score; ``rotary``: rotation of queries and keys; ``kv_from``: the layer whose keys and values this one reads
    instead of having its own; ``pool``: beside its window a query sees one key and value, their means, for each block of so many
    positions (counted from 0) that lies wholly ahead of the window (``None``: nothing ahead of it)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: float = 1.0
    window: int | None = None
    rotary: RotarySpec | None = None
    kv_from: int | None = None
    chunk: int | None = None
    distance_bias: bool = False
    pool: int | None = None

    def validate(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError("AttentionSpec: %d heads of %d / %d over %d key/value heads" % (self.heads, self.dim, self.vdim, self.kv_heads))
        if not self.temp_every > 0:
            raise ValueError("AttentionSpec: temp_every must be positive")
        if self.window is not None and self.window < 1:
            raise ValueError("AttentionSpec: window must be positive or absent")
        if self.chunk is not None and self.chunk < 1:
            raise ValueError("AttentionSpec: chunk must be positive or absent")
        if self.pool is not None and (self.pool < 1 or self.window is None or self.chunk is not None or self.distance_bias):
            raise ValueError("AttentionSpec: pooled blocks of %d positions need a window, and neither chunks nor a distance bias" % self.pool)
        if self.rotary is not None and (self.rotary.dims % 2 or not 0 < self.rotary.dims <= self.dim or self.rotary.base <= 1):
            raise ValueError("AttentionSpec: rotation of %d elements of %d" % (self.rotary.dims, self.dim))

    @property
    def padded_dim(self) -> int:
        return round_up(self.dim, 16)

    @property
    def padded_vdim(self) -> int:
        return round_up(self.vdim, 16)


class DynamicTanh(nn.Module):
    """``tanh(alpha x) * w + b``: a norm without a statistic of the row.  Parameters stay fp32 whatever the model's type."""

    def __init__(self, hidden_size: int):
        super().__init__()
        self.register_buffer("alpha", torch.ones(()))
        self.register_buffer("weight", torch.zeros(round_up(hidden_size, 8)))
        self.register_buffer("bias", torch.zeros(round_up(hidden_size, 8)))
        self.weight[:hidden_size] = 1.0

    def load(self, alpha: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor) -> None:
        n = self.weight.numel()
        self.alpha.copy_(alpha.reshape(()).float())
        self.weight.copy_(pad_to(weight.float(), n))
        self.bias.copy_(pad_to(bias.float(), n))

    def as_epilogue(self, scale: float = 1.0) -> tuple:
        """The parameters in the form that the kernels which end in this norm take."""
        return self.alpha, self.weight, self.bias, scale

    def forward(self, x: torch.Tensor, *, scale: float = 1.0, out_dtype: torch.dtype | None = None) -> torch.Tensor:
        return F.dynamic_tanh(x, self.alpha, self.weight, self.bias, scale=scale, out_dtype=out_dtype)


class PackedParallelBlock(nn.Module):
    """Attention and feed-forward in parallel on one input: ``x += W_o gate(attention(h)) + W_down act(W_up h)``.

    ``qk_norm``: RMS norm of the whole query and key projections (all heads at once); ``head_gate``: one sigmoid gate per
    head from ``h``; ``ff`` ``None``: no feed-forward."""

    def __init__(self, hidden_size: int, attn: AttentionSpec, ff: int | None, activation: str = "gelu", eps: float = 1e-5,
                 qk_norm: bool = True, head_gate: bool = True):
        super().__init__()
        self.attn, self.ff, self.activation, self.eps = attn, ff, activation, eps
        self.qk_norm, self.head_gate = qk_norm, head_gate
        self.hidden_size, width = hidden_size, round_up(hidden_size, 8)
        a = attn
        sizes = (a.heads * a.padded_dim, a.kv_heads * a.padded_dim, a.kv_heads * a.padded_vdim, round_up(ff or 0, 8),
                 round_up(a.heads, 8) if head_gate else 0)
        at, self.segments = 0, []
        for n in sizes:
            self.segments.append((at, n))
            at += n
        self.value_width = a.heads * a.padded_vdim
        self.register_buffer("in_proj", torch.zeros(at, width))
        self.register_buffer("out_proj", torch.zeros(width, self.value_width + sizes[3]))
        self.register_buffer("q_norm", torch.zeros(sizes[0]) if qk_norm else None)
        self.register_buffer("k_norm", torch.zeros(sizes[1]) if qk_norm else None)

    def load(self, q, k, v, o, up=None, down=None, gate=None, q_norm=None, k_norm=None) -> None:
        """Weights as ``[out, in]`` matrices of the true sizes."""
        a, W = self.attn, self.hidden_size
        H, G = a.heads, a.kv_heads
        want = {"q": (q, (H * a.dim, W)), "k": (k, (G * a.dim, W)), "v": (v, (G * a.vdim, W)), "o": (o, (W, H * a.vdim))}
        if self.ff:
            want.update(up=(up, (self.ff, W)), down=(down, (W, self.ff)))
        if self.head_gate:
            want.update(gate=(gate, (H, W)))
        if self.qk_norm:
            want.update(q_norm=(q_norm, (H * a.dim,)), k_norm=(k_norm, (G * a.dim,)))
        for name, (t, shape) in want.items():
            if t is None or tuple(t.shape) != shape:
                raise ValueError("PackedParallelBlock: %s must have shape %s, got %s" % (name, shape, None if t is None else tuple(t.shape)))
        (qo, qn), (ko, kn), (vo, vn), (uo, un), (go, gn) = self.segments
        width = self.in_proj.shape[1]
        for off, n, w in ((qo, qn, pad_heads(q, H, a.padded_dim)), (ko, kn, pad_heads(k, G, a.padded_dim)),
                          (vo, vn, pad_heads(v, G, a.padded_vdim)), (uo, un, up if self.ff else None),
                          (go, gn, gate if self.head_gate else None)):
            if n:
                self.in_proj[off:off + n].copy_(pad_to(w, n, width))
        self.out_proj[:, :self.value_width].copy_(pad_to(pad_heads(o.t(), H, a.padded_vdim).t(), width, self.value_width))
        if self.ff:
            self.out_proj[:, self.value_width:].copy_(pad_to(down, width, un))
        if self.qk_norm:
            self.q_norm.copy_(pad_heads(q_norm.float(), H, a.padded_dim))
            self.k_norm.copy_(pad_heads(k_norm.float(), G, a.padded_dim))

    def unpack(self) -> dict:
        """The inverse of :meth:`load`: views and copies of the true sizes."""
        a, W = self.attn, self.hidden_size
        (qo, qn), (ko, kn), (vo, vn), (uo, un), (go, gn) = self.segments

        def heads(t, n, d):
            return t.unflatten(0, (n, -1))[:, :d].flatten(0, 1)

        w = self.in_proj[:, :W]
        out = {"q": heads(w[qo:qo + qn], a.heads, a.dim), "k": heads(w[ko:ko + kn], a.kv_heads, a.dim), "v": heads(w[vo:vo + vn], a.kv_heads, a.vdim),
               "o": heads(self.out_proj[:W, :self.value_width].t(), a.heads, a.vdim).t()}
        if self.ff:
            out.update(up=w[uo:uo + self.ff], down=self.out_proj[:W, self.value_width:self.value_width + self.ff])
        if self.head_gate:
            out.update(gate=w[go:go + a.heads])
        if self.qk_norm:
            out.update(q_norm=heads(self.q_norm, a.heads, a.dim), k_norm=heads(self.k_norm, a.kv_heads, a.dim))
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        """Random weights of the true sizes (benchmarks and smoke tests)."""
        a, W = self.attn, self.hidden_size
        H, G = a.heads, a.kv_heads

        def rnd(*shape):
            return torch.randn(shape, device=self.in_proj.device, generator=generator) * std

        self.load(rnd(H * a.dim, W), rnd(G * a.dim, W), rnd(G * a.vdim, W), rnd(W, H * a.vdim),
                  *((rnd(self.ff, W), rnd(W, self.ff)) if self.ff else (None, None)), rnd(H, W) if self.head_gate else None,
                  *((torch.ones(H * a.dim), torch.ones(G * a.dim)) if self.qk_norm else (None, None)))

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; norm weights stay fp32."""
        self.in_proj, self.out_proj = self.in_proj.to(dtype), self.out_proj.to(dtype)

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch, cache, layer: int, next_norm: tuple | None = None):
        """Adds the layer to the fp32 residual ``x [T, width]`` in place; returns the next layer's input when
        ``next_norm`` (a :meth:`DynamicTanh.as_epilogue`) is given."""
        a, T = self.attn, h.shape[0]
        seg_q, seg_k, seg_v, seg_up, seg_gate = self.segments
        packed = F.linear_rows(h, self.in_proj)
        acts = torch.empty((T, self.out_proj.shape[1]), device=h.device, dtype=h.dtype)
        F.qkv_finish(packed, cache, layer, batch, q=seg_q, k=seg_k, v=seg_v, up=seg_up, q_weight=self.q_norm, k_weight=self.k_norm,
                     q_count=a.heads * a.dim, k_count=a.kv_heads * a.dim, eps=self.eps, temp_coef=a.temp_coef, temp_every=a.temp_every,
                     act_out=acts[:, self.value_width:], activation=self.activation)
        gate = packed[:, seg_gate[0]:seg_gate[0] + a.heads] if self.head_gate else None
        cache.attend(layer, packed[:, seg_q[0]:seg_q[0] + seg_q[1]].unflatten(1, (a.heads, a.padded_dim)), batch, a.scale, gate=gate,
                     out=acts[:, :self.value_width].unflatten(1, (a.heads, a.padded_vdim)))
        return F.residual_linear_(x, acts, self.out_proj, next_norm)

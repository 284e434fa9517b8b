"""Latent attention over a paged cache: per token a latent of a few hundred elements and one rotated key part are cached;
keys and values of all heads are linear in the latent.

Sizes are padded at load time with zero weights like those of :mod:`~ferrotorch_b200.nn.packed_block`."""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from .. import _native
from ..ops import decoder as D
from ..ops import functional as F
from .gated_attention import checked, unpad_heads
from .packed_block import RotarySpec, pad_heads, pad_to, round_up
from .paged import prefill_pages

FORMED_PAGE = 128    # rows of a page of formed keys
ABSORB_ROWS = 16     # a step whose portions have at most so many tokens treats their rows like single tokens


@dataclass
class LatentSpec:
    """``heads`` query heads with ``dim`` unrotated and ``rot_dim`` rotated elements, values of ``vdim``, a latent of ``rank``;
    ``score = (q . k + q_rot . k_rot) * scale``."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    rotary: RotarySpec

    def validate(self) -> None:
        if min(self.heads, self.dim, self.rot_dim, self.vdim, self.rank) < 1:
            raise ValueError("LatentSpec: %d heads of %d + %d / %d over a latent of %d" % (self.heads, self.dim, self.rot_dim, self.vdim, self.rank))
        r = self.rotary
        if r.dims % 2 or not 0 < r.dims <= self.rot_dim or r.base <= 0 or not r.interleaved:
            raise ValueError("LatentSpec: rotation of %d elements of %d (pairs of neighbours)" % (r.dims, self.rot_dim))

    # a query head is [unrotated | rotated], a cached row [latent | rotated]
    @property
    def padded_dim(self) -> int:
        return round_up(self.dim, 8)

    @property
    def padded_rot(self) -> int:
        return round_up(self.rot_dim, 16)

    @property
    def head_size(self) -> int:
        return round_up(self.padded_dim + self.padded_rot, 16)

    @property
    def padded_vdim(self) -> int:
        return round_up(self.vdim, 16)

    @property
    def padded_rank(self) -> int:
        return round_up(self.rank, 16)

    @property
    def row_size(self) -> int:
        return self.padded_rank + self.padded_rot


class LatentAttention(nn.Module):
    """``W_o (attention(h) * sigmoid(W_g h))``, element by element.

    One packed product ``[q | latent, rotated key | g]`` and one pass for norm, rotation and cache.  Then, for single tokens, short
    portions and in fp32: queries are brought into the latent space (``W_uk`` applied to them instead of to every key), so that all
    heads attend to the cached rows themselves, and the gated product with ``W_uv`` follows.  For longer portions: keys and values of
    their contexts are formed from the cached rows by one product each (the rotated key part passes through it by a unit
    matrix), and the portions run on the prefill kernel, gate included."""

    def __init__(self, hidden_size: int, spec: LatentSpec, eps: float):
        super().__init__()
        self.spec, self.hidden_size, self.eps = spec, hidden_size, eps
        s, width = spec, round_up(hidden_size, 8)
        self.q_width, self.value_width = s.heads * s.head_size, s.heads * s.padded_vdim
        self.register_buffer("in_proj", torch.zeros(self.q_width + s.row_size + self.value_width, width))
        self.register_buffer("latent_norm", torch.zeros(s.padded_rank))
        self.register_buffer("to_latent", torch.zeros(s.heads, 1, s.padded_rank, s.padded_dim))      # W_uk of a head, transposed
        self.register_buffer("to_value", torch.zeros(s.heads, 1, s.padded_vdim, s.padded_rank))      # W_uv of a head
        self.register_buffer("out_proj", torch.zeros(width, self.value_width))
        self.register_buffer("key_proj", None, persistent=False)         # all heads' keys and values from a cached row
        self.register_buffer("value_proj", None, persistent=False)

    def _form_keys(self) -> None:
        s, t = self.spec, self.to_latent
        if t.dtype != torch.bfloat16 or s.head_size > 128 or s.padded_vdim > 128:
            return
        key = torch.zeros(s.heads, s.head_size, s.row_size, dtype=t.dtype, device=t.device)
        key[:, :s.padded_dim, :s.padded_rank] = t[:, 0].transpose(1, 2)
        unit = torch.arange(s.rot_dim, device=t.device)
        key[:, s.padded_dim + unit, s.padded_rank + unit] = 1.0
        self.key_proj = key.flatten(0, 1)
        self.value_proj = pad_to(self.to_value[:, 0].flatten(0, 1), self.value_width, s.row_size)

    def _shapes(self) -> dict:
        W, s = self.hidden_size, self.spec
        return {"q": (s.heads * (s.dim + s.rot_dim), W), "dkv": (s.rank + s.rot_dim, W), "dkv.norm": (s.rank,), "uk": (s.heads * s.dim, s.rank),
                "uv": (s.heads * s.vdim, s.rank), "g": (s.heads * s.vdim, W), "o": (W, s.heads * s.vdim)}

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        """Weights by name (:meth:`tensor_names`), matrices ``[out, in]`` of the true sizes."""
        for name, shape in self._shapes().items():
            checked("LatentAttention", name, sd.get(name), shape)
        s, W, width = self.spec, self.hidden_size, self.in_proj.shape[1]
        q = torch.zeros(s.heads, s.head_size, width, dtype=self.in_proj.dtype, device=self.in_proj.device)
        split = sd["q"].unflatten(0, (s.heads, s.dim + s.rot_dim))
        q[:, :s.dim, :W] = split[:, :s.dim]
        q[:, s.padded_dim:s.padded_dim + s.rot_dim, :W] = split[:, s.dim:]
        row = torch.zeros(s.row_size, width, dtype=self.in_proj.dtype, device=self.in_proj.device)
        row[:s.rank, :W] = sd["dkv"][:s.rank]
        row[s.padded_rank:s.padded_rank + s.rot_dim, :W] = sd["dkv"][s.rank:]
        at = self.q_width + s.row_size
        self.in_proj[:self.q_width].copy_(q.flatten(0, 1))
        self.in_proj[self.q_width:at].copy_(row)
        self.in_proj[at:].copy_(pad_to(pad_heads(sd["g"], s.heads, s.padded_vdim), self.value_width, width))
        self.latent_norm.copy_(pad_to(sd["dkv.norm"].float(), s.padded_rank))
        uk, uv = sd["uk"].unflatten(0, (s.heads, s.dim)), sd["uv"].unflatten(0, (s.heads, s.vdim))
        self.to_latent[:, 0].copy_(pad_to(uk.transpose(1, 2), s.heads, s.padded_rank, s.padded_dim))
        self.to_value[:, 0].copy_(pad_to(uv, s.heads, s.padded_vdim, s.padded_rank))
        self.out_proj.copy_(pad_to(pad_heads(sd["o"].t(), s.heads, s.padded_vdim).t(), width, self.value_width))
        self._form_keys()

    def unpack(self) -> dict:
        s, W = self.spec, self.hidden_size
        q = self.in_proj[:self.q_width, :W].unflatten(0, (s.heads, s.head_size))
        row = self.in_proj[self.q_width:self.q_width + s.row_size, :W]
        return {"q": torch.cat([q[:, :s.dim], q[:, s.padded_dim:s.padded_dim + s.rot_dim]], 1).flatten(0, 1),
                "dkv": torch.cat([row[:s.rank], row[s.padded_rank:s.padded_rank + s.rot_dim]]), "dkv.norm": self.latent_norm[:s.rank],
                "uk": self.to_latent[:, 0, :s.rank, :s.dim].transpose(1, 2).flatten(0, 1), "uv": self.to_value[:, 0, :s.vdim, :s.rank].flatten(0, 1),
                "g": unpad_heads(self.in_proj[self.q_width + s.row_size:, :W], s.heads, s.vdim),
                "o": unpad_heads(self.out_proj[:W].t(), s.heads, s.vdim).t()}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        dev = self.in_proj.device
        self.load({n: torch.ones(s, device=dev) if n.endswith("norm") else torch.randn(s, device=dev, generator=generator) * std
                   for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; the latent's norm weight stays fp32."""
        for name in ("in_proj", "to_latent", "to_value", "out_proj"):
            setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, h: torch.Tensor, batch, cache, layer: int) -> D.SublayerTerms:
        """The sublayer's output for input ``h``; ``layer``: its place in the cache."""
        s, T = self.spec, h.shape[0]
        packed = F.linear_rows(h, self.in_proj)
        formed = self.key_proj is not None and h.is_cuda and s.scale > 0 and batch.longest > ABSORB_ROWS
        n = batch.n_single if formed else T               # rows that attend in the latent space
        q_lat = torch.empty((n, s.heads, s.row_size), device=h.device, dtype=h.dtype)
        D.latent_finish(packed, cache, layer, batch, heads=s.heads, q_off=0, q_head=s.head_size, q_rot=s.padded_dim, c_off=self.q_width,
                        rank=s.rank, rank_pad=s.padded_rank, weight=self.latent_norm, eps=self.eps, table=cache.rotary_table(s.rotary), q_lat=q_lat)
        heads = torch.empty((T, self.value_width), device=h.device, dtype=h.dtype)
        gate = packed[:, self.q_width + s.row_size:]
        if n:
            D.block_linear(packed[:n, :self.q_width], self.to_latent, q_lat.flatten(1), a_col=s.head_size, out_col=s.row_size)
            o_lat = cache.decode(layer, q_lat, batch.visible[:n], s.scale, seq_ids=batch.slots[:n]) if formed else cache.attend(layer, q_lat, batch, s.scale)
            D.block_linear(o_lat.flatten(1), self.to_value, heads[:n], gate=gate[:n])
        if formed:
            q, g, out = (t.unflatten(1, (s.heads, -1)) for t in (packed[:, :self.q_width], gate, heads))
            for rows, spans, longest, table, items in batch.contexts(int(_native.kernels().ft_paged_prefill_tile(1)), FORMED_PAGE):
                ctx = torch.empty((rows, s.row_size), device=h.device, dtype=h.dtype)
                cache.gather_contexts(layer, spans, longest, ctx, FORMED_PAGE)
                k, v = F.linear_rows(ctx, self.key_proj), F.linear_rows(ctx, self.value_proj)
                prefill_pages(q, k.view(-1, FORMED_PAGE, s.heads, s.head_size), v.view(-1, FORMED_PAGE, s.heads, s.padded_vdim), table, items, s.scale,
                              out=out, gate=g)
        return D.SublayerTerms(dense=F.linear_rows(heads, self.out_proj))

"""Recurrent sublayers of decoders: a gated branch, a short causal convolution and a real-gated linear recurrence with
diagonal state, whose sequences live in the slots of an :class:`RGLRUState`; sizes and state of matrix memories
(:class:`MatrixMemorySpec`, :class:`MatrixMemoryState`), which :mod:`~ferrotorch_b200.nn.parallel_mixer` runs beside attention."""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import decoder as D
from ..ops import functional as F
from .gated_attention import checked, unpad_heads
from .packed_block import pad_heads, pad_to, round_up


@dataclass
class RGLRUSpec:
    """``width`` channels in ``blocks`` equal blocks (the gates' matrices are block-diagonal), convolution over ``conv``
    positions, decay ``exp(-decay_scale r softplus(lam))``."""
    width: int
    blocks: int
    conv: int
    decay_scale: float = 8.0

    def validate(self) -> None:
        if min(self.width, self.blocks, self.conv) < 1 or self.width % self.blocks:
            raise ValueError("RGLRUSpec: %d channels in %d blocks, convolution of %d" % (self.width, self.blocks, self.conv))

    @property
    def block(self) -> int:
        return self.width // self.blocks

    @property
    def padded_width(self) -> int:
        return self.blocks * round_up(self.block, 8)


class RGLRUState:
    """State of one layer for every sequence slot: ``state [slots, C]`` fp32 and the last inputs of the convolution
    ``conv [slots, taps - 1, C]`` in the model's type.  A slot is not cleared between sequences: position 0 starts from zero."""

    def __init__(self, slots: int, spec: RGLRUSpec, device, dtype: torch.dtype):
        self.state = torch.zeros((slots, spec.padded_width), device=device, dtype=torch.float32)
        self.conv = torch.zeros((slots, spec.conv - 1, spec.padded_width), device=device, dtype=dtype)


@dataclass
class MatrixMemorySpec:
    """``heads`` memories of ``dim x vdim`` with exponential gates, whose logarithms are capped at ``gate_cap``."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def validate(self) -> None:
        if min(self.heads, self.dim, self.vdim) < 1 or not self.gate_cap > 0:
            raise ValueError("MatrixMemorySpec: %d heads of %d x %d, gates capped at %g" % (self.heads, self.dim, self.vdim, self.gate_cap))

    @property
    def padded_dim(self) -> int:
        return round_up(self.dim, 16)

    @property
    def padded_vdim(self) -> int:
        return round_up(self.vdim, 16)


class MatrixMemoryState:
    """State of one layer for every sequence slot, fp32: the memories ``S [slots, heads, dim, vdim]``, their normalisers ``n [slots,
    heads, dim]`` and the running maxima ``m [slots, heads]`` that both are relative to (padded sizes).  A slot is not cleared between
    sequences: position 0 starts from zero."""

    def __init__(self, slots: int, spec: MatrixMemorySpec, device):
        self.S = torch.zeros((slots, spec.heads, spec.padded_dim, spec.padded_vdim), device=device)
        self.n = torch.zeros((slots, spec.heads, spec.padded_dim), device=device)
        self.m = torch.zeros((slots, spec.heads), device=device)


class RGLRUBlock(nn.Module):
    """``x += W_o (S * gelu(W_y h + b_y))`` with ``S`` the recurrence over ``u = conv(W_x h + b_x)``.

    Two packed products around the convolution, the product of the gates (whose epilogue computes decay and input term, and
    for single tokens the whole step) and the scan over portions."""

    def __init__(self, hidden_size: int, spec: RGLRUSpec):
        super().__init__()
        self.spec, self.hidden_size = spec, hidden_size
        C, n, width = spec.padded_width, round_up(spec.block, 8), round_up(hidden_size, 8)
        self.register_buffer("in_proj", torch.zeros(2 * C, width))            # [y | x]
        self.register_buffer("in_bias", torch.zeros(2 * C))
        self.register_buffer("conv_weight", torch.zeros(spec.conv, C))
        self.register_buffer("conv_bias", torch.zeros(C))
        self.register_buffer("gates", torch.zeros(spec.blocks, 2, n, n))      # recurrence gate, input gate
        self.register_buffer("r_bias", torch.zeros(C))
        self.register_buffer("i_bias", torch.zeros(C))
        self.register_buffer("lam", torch.zeros(C))
        self.register_buffer("decay", torch.zeros(C))
        self.register_buffer("out_proj", torch.zeros(width, C))

    def _shapes(self) -> dict:
        s, W, w = self.spec, self.hidden_size, self.spec.width
        return {"y": (w, W), "y.b": (w,), "x": (w, W), "x.b": (w,), "conv": (w, s.conv), "conv.b": (w,), "ra": (s.blocks, s.block, s.block),
                "ra.b": (s.blocks, s.block), "ri": (s.blocks, s.block, s.block), "ri.b": (s.blocks, s.block), "lam": (w,), "o": (W, w)}

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        s, n = self.spec, round_up(self.spec.block, 8)
        for name, shape in self._shapes().items():
            checked("RGLRUBlock", name, sd.get(name), shape)

        def pad(t):
            return pad_heads(t, s.blocks, n)

        C, width = s.padded_width, self.in_proj.shape[1]
        for i, name in enumerate(("y", "x")):
            self.in_proj[i * C:(i + 1) * C].copy_(pad_to(pad(sd[name]), C, width))
            self.in_bias[i * C:(i + 1) * C].copy_(pad(sd[name + ".b"].float()))
        self.conv_weight.copy_(pad(sd["conv"].float()).t())
        self.conv_bias.copy_(pad(sd["conv.b"].float()))
        for i, name in enumerate(("ra", "ri")):
            self.gates[:, i].copy_(pad_to(sd[name], s.blocks, n, n))
        self.r_bias.copy_(pad(sd["ra.b"].float().flatten()))
        self.i_bias.copy_(pad(sd["ri.b"].float().flatten()))
        self.lam.copy_(pad(sd["lam"].float()))
        self.decay.copy_(-s.decay_scale * torch.nn.functional.softplus(self.lam.double(), threshold=1e9))
        self.out_proj.copy_(pad_to(pad(sd["o"].t()).t(), width, C))

    def unpack(self) -> dict:
        s, W, C = self.spec, self.hidden_size, self.spec.padded_width

        def cut(t):
            return unpad_heads(t, s.blocks, s.block)

        return {"y": cut(self.in_proj[:C, :W]), "y.b": cut(self.in_bias[:C]), "x": cut(self.in_proj[C:, :W]), "x.b": cut(self.in_bias[C:]),
                "conv": cut(self.conv_weight.t()), "conv.b": cut(self.conv_bias), "ra": self.gates[:, 0, :s.block, :s.block],
                "ra.b": cut(self.r_bias).view(s.blocks, -1), "ri": self.gates[:, 1, :s.block, :s.block],
                "ri.b": cut(self.i_bias).view(s.blocks, -1), "lam": cut(self.lam), "o": cut(self.out_proj[:W].t()).t()}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        dev = self.in_proj.device
        self.load({n: torch.randn(s, device=dev, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; convolution, biases and decay stay fp32."""
        for name in ("in_proj", "gates", "out_proj"):
            setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch, state: RGLRUState) -> None:
        """Adds the sublayer of input ``h`` to the fp32 residual ``x`` and carries ``state`` on."""
        C = self.spec.padded_width
        packed = F.linear_rows(h, self.in_proj, self.in_bias)
        y, cx = packed[:, :C], packed[:, C:]
        u = D.causal_conv(cx, self.conv_weight, self.conv_bias, state.conv, batch)
        out = torch.empty((h.shape[0], C), device=h.device, dtype=h.dtype)
        D.gated_recurrence(u, y, self.gates, self.r_bias, self.i_bias, self.decay, state.state, batch, cx, state.conv, out)
        F.residual_linear_(x, out, self.out_proj)

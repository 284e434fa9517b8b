"""Recurrent sublayers of decoders, whose sequences live in the slots of a state: a gated branch, a short causal convolution and a
real-gated linear recurrence with diagonal state (:class:`RGLRUBlock`); a short convolution and state-space heads
(:class:`StateSpaceBlock`); sizes and state of matrix memories (:class:`MatrixMemorySpec`, :class:`MatrixMemoryState`), which
:mod:`~ferrotorch_b200.nn.parallel_mixer` runs beside attention."""
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


@dataclass
class StateSpaceSpec:
    """``heads`` of ``vdim`` elements with states of ``state x vdim``, whose input and output vectors are shared by the heads of each of
    ``groups`` groups; convolution over ``conv`` positions; the gated result is normed in ``norm_groups`` equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int = 1

    def validate(self) -> None:
        if min(self.heads, self.vdim, self.state, self.groups, self.conv, self.norm_groups) < 1 or self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError("StateSpaceSpec: %d heads of %d in %d groups of states of %d, convolution of %d, norm in %d parts"
                             % (self.heads, self.vdim, self.groups, self.state, self.conv, self.norm_groups))

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def padded_vdim(self) -> int:
        return round_up(self.vdim, 16)

    @property
    def padded_state(self) -> int:
        return round_up(self.state, 16)

    @property
    def padded_inner(self) -> int:
        return self.heads * self.padded_vdim

    @property
    def channels(self) -> int:
        """Channels of the convolution (padded)."""
        return self.padded_inner + 2 * self.groups * self.padded_state


class StateSpaceState:
    """State of one layer for every sequence slot: ``S [slots, heads, state, vdim]`` fp32 and the last inputs of the convolution ``conv
    [slots, taps - 1, channels]`` in the model's type (padded sizes).  A slot is not cleared between sequences: position 0 starts
    from zero."""

    def __init__(self, slots: int, spec: StateSpaceSpec, device, dtype: torch.dtype):
        self.S = torch.zeros((slots, spec.heads, spec.padded_state, spec.padded_vdim), device=device)
        self.conv = torch.zeros((slots, spec.conv - 1, spec.channels), device=device, dtype=dtype)


class StateSpaceBlock(nn.Module):
    """State-space duality (Mamba-2): ``W_o (norm(y silu(z)) w)``, ``y`` the heads' states read by C plus ``skip x``, where ``z | x | B | C |
    dt`` is one projection of h and ``x | B | C`` pass a short causal convolution and silu.

    One packed product ``[x | B | C | z | r]`` and one with fp32 results for the step sizes, the convolution, the heads with the gate in
    their epilogue, the norm in place and the output product.  ``residual_gate``: as in
    :class:`~ferrotorch_b200.nn.gated_attention.GatedAttention`."""

    def __init__(self, hidden_size: int, spec: StateSpaceSpec, eps: float, residual_gate: bool = False):
        super().__init__()
        self.spec, self.hidden_size, self.eps, self.residual_gate = spec, hidden_size, eps, residual_gate
        C, inner, width = spec.channels, spec.padded_inner, round_up(hidden_size, 8)
        self.gate_at = C + inner
        self.register_buffer("in_proj", torch.zeros(C + inner + (width if residual_gate else 0), width))
        self.register_buffer("in_bias", torch.zeros(self.in_proj.shape[0]) if residual_gate else None)
        self.register_buffer("step_proj", torch.zeros(round_up(spec.heads, 8), width))
        self.register_buffer("step_bias", torch.zeros(spec.heads))
        self.register_buffer("log_rate", torch.zeros(spec.heads))
        self.register_buffer("rate", torch.ones(spec.heads))
        self.register_buffer("skip", torch.zeros(spec.heads))
        self.register_buffer("conv_weight", torch.zeros(spec.conv, C))
        self.register_buffer("conv_bias", torch.zeros(C))
        self.register_buffer("norm", torch.zeros(inner))
        self.register_buffer("out_proj", torch.zeros(width, inner))

    def _shapes(self) -> dict:
        s, W = self.spec, self.hidden_size
        conv = s.inner + 2 * s.groups * s.state
        out = {"in": (s.inner + conv + s.heads, W), "conv": (conv, s.conv), "conv.b": (conv,), "dt_bias": (s.heads,), "A_log": (s.heads,),
               "D": (s.heads,), "norm": (s.inner,), "o": (W, s.inner)}
        if self.residual_gate:
            out.update({"rg": (W, W), "rg.b": (W,)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def _pad_conv(self, t: torch.Tensor) -> torch.Tensor:
        """Rows ``[x | B | C]`` padded."""
        s = self.spec
        x, b, c = t.split([s.inner, s.groups * s.state, s.groups * s.state])
        return torch.cat([pad_heads(x, s.heads, s.padded_vdim), pad_heads(b, s.groups, s.padded_state), pad_heads(c, s.groups, s.padded_state)])

    def _cut_conv(self, t: torch.Tensor) -> torch.Tensor:
        s, n = self.spec, self.spec.groups * self.spec.padded_state
        x, b, c = t.split([s.padded_inner, n, n])
        return torch.cat([unpad_heads(x, s.heads, s.vdim), unpad_heads(b, s.groups, s.state), unpad_heads(c, s.groups, s.state)])

    def load(self, sd: dict) -> None:
        """Weights by name (:meth:`tensor_names`), matrices ``[out, in]`` of the true sizes."""
        s = self.spec
        for name, shape in self._shapes().items():
            checked("StateSpaceBlock", name, sd.get(name), shape)
        C, width = s.channels, self.in_proj.shape[1]
        z, xbc, dt = sd["in"].split([s.inner, s.inner + 2 * s.groups * s.state, s.heads])
        self.in_proj[:C].copy_(pad_to(self._pad_conv(xbc), C, width))
        self.in_proj[C:self.gate_at].copy_(pad_to(pad_heads(z, s.heads, s.padded_vdim), s.padded_inner, width))
        if self.residual_gate:
            self.in_proj[self.gate_at:].copy_(pad_to(sd["rg"], width, width))
            self.in_bias[self.gate_at:].copy_(pad_to(sd["rg.b"].float(), width))
        self.step_proj.copy_(pad_to(dt, *self.step_proj.shape))
        self.step_bias.copy_(sd["dt_bias"].float())
        self.log_rate.copy_(sd["A_log"].float())
        self.rate.copy_(self.log_rate.double().exp())
        self.skip.copy_(sd["D"].float())
        self.conv_weight.copy_(self._pad_conv(sd["conv"].float()).t())
        self.conv_bias.copy_(self._pad_conv(sd["conv.b"].float()))
        self.norm.copy_(pad_heads(sd["norm"].float(), s.heads, s.padded_vdim))
        self.out_proj.copy_(pad_to(pad_heads(sd["o"].t(), s.heads, s.padded_vdim).t(), width, s.padded_inner))

    def unpack(self) -> dict:
        s, W, C = self.spec, self.hidden_size, self.spec.channels
        out = {"in": torch.cat([unpad_heads(self.in_proj[C:self.gate_at, :W], s.heads, s.vdim), self._cut_conv(self.in_proj[:C, :W]), self.step_proj[:s.heads, :W]]),
               "conv": self._cut_conv(self.conv_weight.t()), "conv.b": self._cut_conv(self.conv_bias), "dt_bias": self.step_bias, "A_log": self.log_rate,
               "D": self.skip, "norm": unpad_heads(self.norm, s.heads, s.vdim), "o": unpad_heads(self.out_proj[:W].t(), s.heads, s.vdim).t()}
        if self.residual_gate:
            out.update({"rg": self.in_proj[self.gate_at:self.gate_at + W, :W], "rg.b": self.in_bias[self.gate_at:self.gate_at + W]})
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        dev = self.in_proj.device
        self.load({n: torch.ones(s, device=dev) if n in ("norm", "D") else torch.randn(s, device=dev, generator=generator) * std
                   for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; convolution, biases, rates and norm weights stay fp32."""
        for name in ("in_proj", "step_proj", "out_proj"):
            setattr(self, name, getattr(self, name).to(dtype))

    def terms(self, h: torch.Tensor, batch, state: StateSpaceState) -> tuple:
        """The sublayer's output and the pre-activations of its residual gate (a view; ``None`` without one); carries ``state`` on."""
        s, C = self.spec, self.spec.channels
        packed = F.linear_rows(h, self.in_proj, self.in_bias)
        step = D.few_outputs(h, self.step_proj)
        xbc, z = packed[:, :C], packed[:, C:self.gate_at]
        u = D.causal_conv(xbc, self.conv_weight, self.conv_bias, state.conv, batch, silu=True)
        D.conv_tail(xbc, state.conv, batch)
        y = torch.empty((h.shape[0], s.padded_inner), device=h.device, dtype=h.dtype)
        D.state_space(u, z, step, self.step_bias, self.rate, self.skip, state.S, batch, y, heads=s.heads, groups=s.groups)
        D.part_norm_(y, self.norm, s.norm_groups, self.eps, heads=s.heads, vdim=s.vdim)
        return D.SublayerTerms(dense=F.linear_rows(y, self.out_proj)), packed[:, self.gate_at:] if self.residual_gate else None

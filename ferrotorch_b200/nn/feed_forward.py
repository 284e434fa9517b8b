"""Feed-forward sublayers of decoders with an fp32 residual stream: dense, and routed experts."""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..ops import decoder as D
from ..ops import functional as F
from .gated_attention import checked
from .packed_block import pad_to, round_up


class PackedMLP(nn.Module):
    """``W_down act(W_up h)``: added to the residual (:meth:`forward`) or left to the kernel that does (:meth:`terms`).

    ``activation``: one that the GEMM epilogue applies (relu2, relu, silu, gelu in erf form), or ``poly_norm``, a sum of normed powers
    with the coefficients ``act`` (:func:`~ferrotorch_b200.ops.decoder.poly_norm`, ``eps``).  ``residual_gate``: pre-activations of a gate
    of the whole sublayer, ``rg`` with its bias ``rg.b``, from one product with W_up where its epilogue has no activation."""

    def __init__(self, hidden_size: int, ff: int, activation: str = "relu2", eps: float = 1e-5, residual_gate: bool = False):
        super().__init__()
        self.hidden_size, self.ff, self.activation, self.eps, self.residual_gate = hidden_size, ff, activation, eps, residual_gate
        if residual_gate and activation != "poly_norm":
            raise ValueError("PackedMLP: a residual gate beside activation %r" % activation)
        width, n = round_up(hidden_size, 8), round_up(ff, 8)
        self.register_buffer("up", torch.zeros(n + (width if residual_gate else 0), width))
        self.register_buffer("bias", torch.zeros(n + width) if residual_gate else None)
        self.register_buffer("down", torch.zeros(width, n))
        self.register_buffer("act", torch.zeros(4) if activation == "poly_norm" else None)

    def _shapes(self) -> dict:
        W = self.hidden_size
        out = {"up": (self.ff, W), "down": (W, self.ff)}
        if self.act is not None:
            out["act"] = (4,)
        if self.residual_gate:
            out.update({"rg": (W, W), "rg.b": (W,)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def _views(self) -> dict:
        """The (padded) buffer or part of one behind every tensor."""
        n = self.down.shape[1]
        out = {"up": self.up[:n], "down": self.down, "act": self.act}
        if self.residual_gate:
            out.update({"rg": self.up[n:], "rg.b": self.bias[n:]})
        return out

    def load(self, sd: dict) -> None:
        views = self._views()
        for name, shape in self._shapes().items():
            views[name].copy_(pad_to(checked("PackedMLP", name, sd.get(name), shape), *views[name].shape))

    def unpack(self) -> dict:
        views = self._views()
        return {n: views[n][tuple(slice(0, k) for k in s)] for n, s in self._shapes().items()}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        self.load({n: torch.randn(s, device=self.up.device, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; bias and coefficients stay fp32."""
        self.up, self.down = self.up.to(dtype), self.down.to(dtype)

    def forward(self, x: torch.Tensor, h: torch.Tensor) -> None:
        if self.residual_gate:
            raise ValueError("PackedMLP: the residual gate needs the kernel that adds the terms")
        F.residual_linear_(x, self._hidden(h)[0], self.down)

    def _hidden(self, h: torch.Tensor) -> tuple:
        if self.act is None:
            return F.linear_rows(h, self.up, activation=self.activation), None
        n = self.down.shape[1]
        packed = F.linear_rows(h, self.up, self.bias)
        return D.poly_norm(packed[:, :n], self.act, self.eps, count=self.ff), packed[:, n:] if self.residual_gate else None

    def terms(self, h: torch.Tensor) -> tuple:
        """The sublayer's output and the pre-activations of its residual gate (a view; ``None`` without one)."""
        act, gate = self._hidden(h)
        return D.SublayerTerms(dense=F.linear_rows(act, self.down)), gate


@dataclass
class ExpertSpec:
    """``experts`` feed-forward layers of width ``ff``, of which a row uses ``top``: ``W_down (act(W_gate z) * (W_up z))`` when
    ``gated``, else ``W_down act(W_up z)``.

    ``score`` ``sigmoid``: the largest router logits, weighted by their sigmoid; ``softmax``: the largest softmax scores (after adding
    a learned ``correction`` per output, which the weights do not contain).  ``router_bias``: a learned number per output joins the
    logits.  ``normalize``: weights divided by their sum (of softmax scores: the softmax over the chosen alone).  ``scale``: whether a
    weight multiplies the expert's ``input`` or ``output``.  ``identity``: so many more outputs of the router, whose "expert" is the
    input itself.  ``shared_ff``: width of one more expert that every row uses (``None``: none), with weight 1 or, with
    ``shared_gate``, the sigmoid of a product with the row."""
    experts: int
    top: int
    ff: int
    score: str = "sigmoid"
    correction: bool = False
    normalize: bool = False
    scale: str = "input"
    identity: int = 0
    shared_ff: int | None = None
    gated: bool = True
    router_bias: bool = False
    shared_gate: bool = False

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def validate(self) -> None:
        if min(self.experts, self.top, self.ff) < 1 or self.identity < 0 or self.top > self.outputs or self.outputs + self.shared_gate > 1024:
            raise ValueError("ExpertSpec: %d of %d experts (and %d identities) of width %d" % (self.top, self.experts, self.identity, self.ff))
        if self.score not in ("sigmoid", "softmax") or self.scale not in ("input", "output") or (self.correction and self.score != "softmax"):
            raise ValueError("ExpertSpec: score %r with correction %r, scale %r" % (self.score, self.correction, self.scale))
        if self.shared_ff is not None and self.shared_ff < 1:
            raise ValueError("ExpertSpec: the shared expert's width must be positive or absent")
        if self.shared_gate and self.shared_ff is None:
            raise ValueError("ExpertSpec: a gate of the shared expert without one")
        if (self.identity or not self.gated) and self.scale != "output":
            raise ValueError("ExpertSpec: identity experts and experts without a gate need weights on the outputs")


class RoutedExperts(nn.Module):
    """Sum over a row's experts by the rules of an :class:`ExpertSpec`; ``activation``: silu, relu or gelu of gated experts, relu2 of
    the others.

    The result stays with the sorted rows: :meth:`forward` returns :class:`~ferrotorch_b200.ops.decoder.SublayerTerms` for the
    kernel that reads the residual next, which adds them on its way.  ``residual_gate``: pre-activations of a gate of the whole
    sublayer, ``rg`` with its bias ``rg.b`` (:meth:`terms`)."""

    def __init__(self, hidden_size: int, spec: ExpertSpec, activation: str = "silu", residual_gate: bool = False):
        super().__init__()
        self.hidden_size, self.spec, self.activation, self.residual_gate = hidden_size, spec, activation, residual_gate
        if spec.gated == (activation == "relu2"):
            raise ValueError("RoutedExperts: activation %r of experts %s a gate" % (activation, "with" if spec.gated else "without"))
        width, n = round_up(hidden_size, 8), round_up(spec.ff, 8)
        self.register_buffer("router", torch.zeros(round_up(spec.outputs + spec.shared_gate, 8), width))
        self.register_buffer("router_bias", torch.zeros(spec.outputs) if spec.router_bias else None)
        self.register_buffer("correction", torch.zeros(spec.outputs) if spec.correction else None)
        parts = 2 if spec.gated else 1
        self.register_buffer("gate_up", torch.zeros(spec.experts, parts, n, width))
        self.register_buffer("down", torch.zeros(spec.experts, 1, width, n))
        m = round_up(spec.shared_ff or 0, 8)
        self.register_buffer("shared_gate_up", torch.zeros(1, parts, m, width) if m else None)
        self.register_buffer("shared_down", torch.zeros(width, m) if m else None)
        self.register_buffer("residual_proj", torch.zeros(width, width) if residual_gate else None)
        self.register_buffer("residual_bias", torch.zeros(width) if residual_gate else None)

    def _shapes(self) -> dict:
        W, s = self.hidden_size, self.spec
        out = {"router": (s.outputs, W)}
        if s.router_bias:
            out["router.b"] = (s.outputs,)
        if s.correction:
            out["correction"] = (s.outputs,)
        for name, ff in [("e%d" % e, s.ff) for e in range(s.experts)] + ([("shared", s.shared_ff)] if s.shared_ff else []):
            if s.gated:
                out[name + ".gate"] = (ff, W)
            out.update({name + ".up": (ff, W), name + ".down": (W, ff)})
        if s.shared_gate:
            out["shared.sg"] = (1, W)
        if self.residual_gate:
            out.update({"rg": (W, W), "rg.b": (W,)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def _views(self) -> dict:
        """The (padded) buffer or part of one behind every tensor."""
        s, W = self.spec, self.hidden_size
        out = {"router": self.router[:s.outputs], "router.b": self.router_bias, "correction": self.correction,
               "shared.sg": self.router[s.outputs:s.outputs + 1], "rg": self.residual_proj, "rg.b": self.residual_bias}
        parts = ("gate", "up") if s.gated else ("up",)
        for name, ups, down in [("e%d" % e, self.gate_up[e], self.down[e, 0]) for e in range(s.experts)] + (
                [("shared", self.shared_gate_up[0], self.shared_down)] if s.shared_ff else []):
            out.update({"%s.%s" % (name, part): ups[i] for i, part in enumerate(parts)})
            out[name + ".down"] = down
        return out

    def load(self, sd: dict) -> None:
        shapes, views = self._shapes(), self._views()
        for name, shape in shapes.items():
            checked("RoutedExperts", name, sd.get(name), shape)
        for name in shapes:
            views[name].copy_(pad_to(sd[name], *views[name].shape))

    def unpack(self) -> dict:
        views = self._views()
        return {n: views[n][tuple(slice(0, k) for k in s)] for n, s in self._shapes().items()}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        self.load({n: torch.randn(s, device=self.router.device, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; biases and corrections stay fp32."""
        for name in ("router", "gate_up", "down", "shared_gate_up", "shared_down", "residual_proj"):
            if getattr(self, name) is not None:
                setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, h: torch.Tensor) -> D.SublayerTerms:
        s, T = self.spec, h.shape[0]
        route = D.moe_route(h, self.router, s.experts, s.top, identity=s.identity, score=s.score, correction=self.correction, normalize=s.normalize,
                            bias=self.router_bias, gate=s.shared_gate)
        on_input = s.scale == "input"
        if s.gated:
            act = D.grouped_linear(route.sorted, self.gate_up, route, glu=self.activation, seg_rows=T, scaled=on_input)
        else:
            act = D.grouped_linear(route.sorted, self.gate_up, route, seg_rows=T, activation=self.activation)
        terms, dense = D.grouped_linear(act, self.down, route, seg_rows=T), None
        if self.shared_down is not None:
            if s.gated:
                act = torch.empty((T, self.shared_down.shape[1]), device=h.device, dtype=h.dtype)
                D.block_linear(h, self.shared_gate_up, act, glu=self.activation)
            else:
                act = F.linear_rows(h, self.shared_gate_up[0, 0], activation=self.activation)
            dense = F.linear_rows(act, self.shared_down)
        return D.SublayerTerms(terms, route.place, None if on_input else route.weight, dense, h if s.identity else None, route.gate)

    def terms(self, h: torch.Tensor) -> tuple:
        """The sublayer's output and the pre-activations of its residual gate (``None`` without one)."""
        gate = F.linear_rows(h, self.residual_proj, self.residual_bias) if self.residual_gate else None
        return self.forward(h), gate

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
    """``x += W_down act(W_up h)``; ``activation``: one that the GEMM epilogue applies (relu2, relu, silu, gelu in erf form)."""

    def __init__(self, hidden_size: int, ff: int, activation: str = "relu2"):
        super().__init__()
        self.hidden_size, self.ff, self.activation = hidden_size, ff, activation
        width, n = round_up(hidden_size, 8), round_up(ff, 8)
        self.register_buffer("up", torch.zeros(n, width))
        self.register_buffer("down", torch.zeros(width, n))

    def _shapes(self) -> dict:
        return {"up": (self.ff, self.hidden_size), "down": (self.hidden_size, self.ff)}

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        for name, shape in self._shapes().items():
            buf = getattr(self, name)
            buf.copy_(pad_to(checked("PackedMLP", name, sd.get(name), shape), *buf.shape))

    def unpack(self) -> dict:
        return {n: getattr(self, n)[:s[0], :s[1]] for n, s in self._shapes().items()}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        self.load({n: torch.randn(s, device=self.up.device, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        self.up, self.down = self.up.to(dtype), self.down.to(dtype)

    def forward(self, x: torch.Tensor, h: torch.Tensor) -> None:
        F.residual_linear_(x, F.linear_rows(h, self.up, activation=self.activation), self.down)


@dataclass
class ExpertSpec:
    """``experts`` gated feed-forward layers of width ``ff``, of which a row uses the ``top`` with the largest router logits."""
    experts: int
    top: int
    ff: int

    def validate(self) -> None:
        if min(self.experts, self.top, self.ff) < 1 or self.top > self.experts or self.experts > 1024:
            raise ValueError("ExpertSpec: %d of %d experts of width %d" % (self.top, self.experts, self.ff))


class RoutedExperts(nn.Module):
    """Sum over a row's experts of ``expert(w h)``, ``expert(z) = W_down (act(W_gate z) * (W_up z))``, ``w`` the sigmoid of the
    expert's router logit (not renormalised).

    The result stays with the sorted rows: :meth:`forward` returns ``(terms, where)`` for the norm that reads the residual
    next (:func:`~ferrotorch_b200.ops.decoder.rms_rows`), which adds them on its way."""

    def __init__(self, hidden_size: int, spec: ExpertSpec, activation: str = "silu"):
        super().__init__()
        self.hidden_size, self.spec, self.activation = hidden_size, spec, activation
        width, n = round_up(hidden_size, 8), round_up(spec.ff, 8)
        self.register_buffer("router", torch.zeros(round_up(spec.experts, 8), width))
        self.register_buffer("gate_up", torch.zeros(spec.experts, 2, n, width))
        self.register_buffer("down", torch.zeros(spec.experts, 1, width, n))

    def _shapes(self) -> dict:
        W, ff = self.hidden_size, self.spec.ff
        out = {"router": (self.spec.experts, W)}
        for e in range(self.spec.experts):
            out.update({"e%d.gate" % e: (ff, W), "e%d.up" % e: (ff, W), "e%d.down" % e: (W, ff)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        for name, shape in self._shapes().items():
            checked("RoutedExperts", name, sd.get(name), shape)
        self.router.copy_(pad_to(sd["router"], *self.router.shape))
        for e in range(self.spec.experts):
            for buf, name in ((self.gate_up[e, 0], "gate"), (self.gate_up[e, 1], "up"), (self.down[e, 0], "down")):
                buf.copy_(pad_to(sd["e%d.%s" % (e, name)], *buf.shape))

    def unpack(self) -> dict:
        W, ff = self.hidden_size, self.spec.ff
        out = {"router": self.router[:self.spec.experts, :W]}
        for e in range(self.spec.experts):
            out.update({"e%d.gate" % e: self.gate_up[e, 0, :ff, :W], "e%d.up" % e: self.gate_up[e, 1, :ff, :W],
                        "e%d.down" % e: self.down[e, 0, :W, :ff]})
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        self.load({n: torch.randn(s, device=self.router.device, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        for name in ("router", "gate_up", "down"):
            setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, x: torch.Tensor, h: torch.Tensor) -> tuple:
        s, T = self.spec, h.shape[0]
        route = D.moe_route(h, self.router, s.experts, s.top)
        act = D.grouped_linear(route.sorted, self.gate_up, route, glu=self.activation, seg_rows=T)
        return D.grouped_linear(act, self.down, route, seg_rows=T), route.place

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
    """``experts`` gated feed-forward layers of width ``ff``, of which a row uses ``top``.

    ``score`` ``sigmoid``: the largest router logits, weighted by their sigmoid; ``softmax``: the largest softmax scores (after adding
    a learned ``correction`` per output, which the weights do not contain).  ``normalize``: weights divided by their sum.  ``scale``:
    whether a weight multiplies the expert's ``input`` or ``output``.  ``identity``: so many more outputs of the router, whose
    "expert" is the input itself.  ``shared_ff``: width of one more expert that every row uses, with weight 1 (``None``: none)."""
    experts: int
    top: int
    ff: int
    score: str = "sigmoid"
    correction: bool = False
    normalize: bool = False
    scale: str = "input"
    identity: int = 0
    shared_ff: int | None = None

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def validate(self) -> None:
        if min(self.experts, self.top, self.ff) < 1 or self.identity < 0 or self.top > self.outputs or self.outputs > 1024:
            raise ValueError("ExpertSpec: %d of %d experts (and %d identities) of width %d" % (self.top, self.experts, self.identity, self.ff))
        if self.score not in ("sigmoid", "softmax") or self.scale not in ("input", "output") or (self.correction and self.score != "softmax"):
            raise ValueError("ExpertSpec: score %r with correction %r, scale %r" % (self.score, self.correction, self.scale))
        if self.shared_ff is not None and self.shared_ff < 1:
            raise ValueError("ExpertSpec: the shared expert's width must be positive or absent")
        if self.identity and self.scale != "output":
            raise ValueError("ExpertSpec: identity experts need weights on the outputs")


class RoutedExperts(nn.Module):
    """Sum over a row's experts, ``expert(z) = W_down (act(W_gate z) * (W_up z))``, by the rules of an :class:`ExpertSpec`.

    The result stays with the sorted rows: :meth:`forward` returns :class:`~ferrotorch_b200.ops.decoder.SublayerTerms` for the
    kernel that reads the residual next, which adds them on its way."""

    def __init__(self, hidden_size: int, spec: ExpertSpec, activation: str = "silu"):
        super().__init__()
        self.hidden_size, self.spec, self.activation = hidden_size, spec, activation
        width, n = round_up(hidden_size, 8), round_up(spec.ff, 8)
        self.register_buffer("router", torch.zeros(round_up(spec.outputs, 8), width))
        self.register_buffer("correction", torch.zeros(spec.outputs) if spec.correction else None)
        self.register_buffer("gate_up", torch.zeros(spec.experts, 2, n, width))
        self.register_buffer("down", torch.zeros(spec.experts, 1, width, n))
        m = round_up(spec.shared_ff or 0, 8)
        self.register_buffer("shared_gate_up", torch.zeros(1, 2, m, width) if m else None)
        self.register_buffer("shared_down", torch.zeros(width, m) if m else None)

    def _shapes(self) -> dict:
        W, s = self.hidden_size, self.spec
        out = {"router": (s.outputs, W)}
        if s.correction:
            out["correction"] = (s.outputs,)
        for name, ff in [("e%d" % e, s.ff) for e in range(s.experts)] + ([("shared", s.shared_ff)] if s.shared_ff else []):
            out.update({name + ".gate": (ff, W), name + ".up": (ff, W), name + ".down": (W, ff)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def _parts(self) -> list:
        """``(name, gate, up, down)`` of every expert, as views of the packed buffers."""
        out = [("e%d" % e, self.gate_up[e, 0], self.gate_up[e, 1], self.down[e, 0]) for e in range(self.spec.experts)]
        if self.shared_down is not None:
            out.append(("shared", self.shared_gate_up[0, 0], self.shared_gate_up[0, 1], self.shared_down))
        return out

    def load(self, sd: dict) -> None:
        for name, shape in self._shapes().items():
            checked("RoutedExperts", name, sd.get(name), shape)
        self.router.copy_(pad_to(sd["router"], *self.router.shape))
        if self.correction is not None:
            self.correction.copy_(sd["correction"].float())
        for name, gate, up, down in self._parts():
            for buf, part in ((gate, "gate"), (up, "up"), (down, "down")):
                buf.copy_(pad_to(sd["%s.%s" % (name, part)], *buf.shape))

    def unpack(self) -> dict:
        W, shapes = self.hidden_size, self._shapes()
        out = {"router": self.router[:self.spec.outputs, :W]}
        if self.correction is not None:
            out["correction"] = self.correction
        for name, gate, up, down in self._parts():
            for buf, part in ((gate, "gate"), (up, "up"), (down, "down")):
                n, k = shapes["%s.%s" % (name, part)]
                out["%s.%s" % (name, part)] = buf[:n, :k]
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        self.load({n: torch.randn(s, device=self.router.device, generator=generator) * std for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; corrections stay fp32."""
        for name in ("router", "gate_up", "down", "shared_gate_up", "shared_down"):
            if getattr(self, name) is not None:
                setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, h: torch.Tensor) -> D.SublayerTerms:
        s, T = self.spec, h.shape[0]
        route = D.moe_route(h, self.router, s.experts, s.top, identity=s.identity, score=s.score, correction=self.correction, normalize=s.normalize)
        on_input = s.scale == "input"
        act = D.grouped_linear(route.sorted, self.gate_up, route, glu=self.activation, seg_rows=T, scaled=on_input)
        terms, dense = D.grouped_linear(act, self.down, route, seg_rows=T), None
        if self.shared_down is not None:
            act = torch.empty((T, self.shared_down.shape[1]), device=h.device, dtype=h.dtype)
            dense = F.linear_rows(D.block_linear(h, self.shared_gate_up, act, glu=self.activation), self.shared_down)
        return D.SublayerTerms(terms, route.place, None if on_input else route.weight, dense, h if s.identity else None)

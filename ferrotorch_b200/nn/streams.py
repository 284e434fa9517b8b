"""Residuals of several fp32 streams (hyper-connections): every sublayer reads a weighted sum of the streams and leaves its
output in all of them."""
from __future__ import annotations

import torch
from torch import nn

from ..ops import decoder as D
from .gated_attention import checked


class StreamMixing(nn.Module):
    """The connection of one sublayer to ``streams`` residual streams: its input is ``sum_s into[s] x_s``, and with its output y all
    streams become ``x_t <- sum_s mix[s, t] x_s + out[t] y`` at once.  The weights stay fp32 whatever the model's type."""

    def __init__(self, streams: int):
        super().__init__()
        self.streams = streams
        self.register_buffer("into", torch.full((streams,), 1.0 / streams))
        self.register_buffer("out", torch.ones(streams))
        self.register_buffer("mix", torch.eye(streams))

    def _shapes(self) -> dict:
        return {"in": (self.streams,), "out": (self.streams,), "mix": (self.streams, self.streams)}

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        for name, shape in self._shapes().items():
            checked("StreamMixing", name, sd.get(name), shape)
        self.into.copy_(sd["in"].float())
        self.out.copy_(sd["out"].float())
        self.mix.copy_(sd["mix"].float())

    def unpack(self) -> dict:
        return {"in": self.into, "out": self.out, "mix": self.mix}

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        s, dev = self.streams, self.into.device

        def rnd(*shape):
            return torch.randn(shape, device=dev, generator=generator) * std

        self.load({"in": 1.0 / s + rnd(s), "out": 1.0 + rnd(s), "mix": torch.eye(s, device=dev) + rnd(s, s)})

    def step(self, x: torch.Tensor, y: D.SublayerTerms, into: torch.Tensor, norm, out_dtype: torch.dtype, **kw):
        """The streams ``x [T, S, H]`` after this sublayer's output ``y``, and the normed input of the next one, whose weights are
        ``into`` and whose norm is a :class:`~ferrotorch_b200.nn.gated_attention.ResidualRMSNorm`: ``(x', h)``."""
        if norm.offset:
            raise ValueError("StreamMixing: norm weights are stored around zero")
        return D.stream_step(x, y, self.mix, self.out, into, norm.weight, norm.eps, count=norm.hidden_size, out_dtype=out_dtype, **kw)

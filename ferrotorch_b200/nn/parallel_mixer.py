"""Two mixers side by side on one input: chunked attention with a distance bias over a paged cache, and matrix memories whose
sequences live in the slots of a :class:`~ferrotorch_b200.nn.recurrent.MatrixMemoryState`.

Sizes are padded at load time with zero weights like those of :mod:`~ferrotorch_b200.nn.packed_block`."""
from __future__ import annotations

import torch
from torch import nn

from ..ops import decoder as D
from ..ops import functional as F
from .gated_attention import checked, unpad_heads
from .packed_block import AttentionSpec, head_slopes, pad_heads, pad_to, round_up
from .recurrent import MatrixMemorySpec, MatrixMemoryState


class AttentionMemoryMixer(nn.Module):
    """``left_scale * W_o attention(h) + right_scale * W_o' (norm(memory(h)) * sigmoid(W_g h))``.

    One packed product ``[q | k | v | q' | k' | v' | g']`` of both sides and one with fp32 results for the memories' gates; a pass
    that norms queries and keys (RMS per head, no weight) and fills the pages; the attention and the memories, each writing its scaled
    heads into the operand of one output product ``[W_o | W_o']``."""

    def __init__(self, hidden_size: int, attn: AttentionSpec, memory: MatrixMemorySpec, left_scale: float, right_scale: float, eps: float):
        super().__init__()
        if attn.window is not None or attn.rotary is not None or attn.kv_from is not None:
            raise ValueError("AttentionMemoryMixer: attention with a window, rotation or keys of another layer")
        self.attn, self.memory, self.hidden_size, self.eps = attn, memory, hidden_size, eps
        self.left_scale, self.right_scale = left_scale, right_scale
        a, m, width = attn, memory, round_up(hidden_size, 8)
        self.left_width, self.right_width = a.heads * a.padded_vdim, m.heads * m.padded_vdim
        # name, heads, head size, padded head size
        self.parts = [("left.q", a.heads, a.dim, a.padded_dim), ("left.k", a.kv_heads, a.dim, a.padded_dim), ("left.v", a.kv_heads, a.vdim, a.padded_vdim),
                      ("right.q", m.heads, m.dim, m.padded_dim), ("right.k", m.heads, m.dim, m.padded_dim), ("right.v", m.heads, m.vdim, m.padded_vdim),
                      ("right.g", m.heads, m.vdim, m.padded_vdim)]
        at, self.offsets = 0, {}
        for name, heads, _, padded in self.parts:
            self.offsets[name] = at
            at += heads * padded
        self.n_gate = round_up(m.heads, 4)
        self.register_buffer("in_proj", torch.zeros(at, width))
        self.register_buffer("gate_proj", torch.zeros(2 * self.n_gate, width))          # input gates, forget gates
        self.register_buffer("i_bias", torch.zeros(m.heads))
        self.register_buffer("f_bias", torch.zeros(m.heads))
        self.register_buffer("norm", torch.zeros(self.right_width))
        self.register_buffer("out_proj", torch.zeros(width, self.left_width + self.right_width))
        self.register_buffer("ones", torch.ones(a.padded_dim))
        self.register_buffer("slopes", head_slopes(a.heads) if a.distance_bias else None)

    def _shapes(self) -> dict:
        W, a, m = self.hidden_size, self.attn, self.memory
        out = {name: (heads * d, W) for name, heads, d, _ in self.parts}
        out.update({"left.o": (W, a.heads * a.vdim), "right.o": (W, m.heads * m.vdim), "right.norm": (m.heads * m.vdim,), "right.i": (m.heads, W),
                    "right.i.b": (m.heads,), "right.f": (m.heads, W), "right.f.b": (m.heads,)})
        return out

    def tensor_names(self) -> list:
        return list(self._shapes())

    def load(self, sd: dict) -> None:
        """Weights by name (:meth:`tensor_names`), matrices ``[out, in]`` of the true sizes."""
        for name, shape in self._shapes().items():
            checked("AttentionMemoryMixer", name, sd.get(name), shape)
        a, m, width = self.attn, self.memory, self.in_proj.shape[1]
        for name, heads, _, padded in self.parts:
            at, n = self.offsets[name], heads * padded
            self.in_proj[at:at + n].copy_(pad_to(pad_heads(sd[name], heads, padded), n, width))
        self.gate_proj[:m.heads].copy_(pad_to(sd["right.i"], m.heads, width))
        self.gate_proj[self.n_gate:self.n_gate + m.heads].copy_(pad_to(sd["right.f"], m.heads, width))
        self.i_bias.copy_(sd["right.i.b"].float())
        self.f_bias.copy_(sd["right.f.b"].float())
        self.norm.copy_(pad_heads(sd["right.norm"].float(), m.heads, m.padded_vdim))
        self.out_proj[:, :self.left_width].copy_(pad_to(pad_heads(sd["left.o"].t(), a.heads, a.padded_vdim).t(), width, self.left_width))
        self.out_proj[:, self.left_width:].copy_(pad_to(pad_heads(sd["right.o"].t(), m.heads, m.padded_vdim).t(), width, self.right_width))

    def unpack(self) -> dict:
        a, m, W = self.attn, self.memory, self.hidden_size
        out = {name: unpad_heads(self.in_proj[self.offsets[name]:self.offsets[name] + heads * padded, :W], heads, d)
               for name, heads, d, padded in self.parts}
        out.update({"left.o": unpad_heads(self.out_proj[:W, :self.left_width].t(), a.heads, a.vdim).t(),
                    "right.o": unpad_heads(self.out_proj[:W, self.left_width:].t(), m.heads, m.vdim).t(),
                    "right.norm": unpad_heads(self.norm, m.heads, m.vdim), "right.i": self.gate_proj[:m.heads, :W], "right.i.b": self.i_bias,
                    "right.f": self.gate_proj[self.n_gate:self.n_gate + m.heads, :W], "right.f.b": self.f_bias})
        return out

    def random_(self, std: float, generator: torch.Generator | None = None) -> None:
        dev = self.in_proj.device
        self.load({n: torch.ones(s, device=dev) if n.endswith("norm") else torch.randn(s, device=dev, generator=generator) * std
                   for n, s in self._shapes().items()})

    def cast_(self, dtype: torch.dtype) -> None:
        """The matrices in ``dtype``; biases, norm weights and slopes stay fp32."""
        for name in ("in_proj", "gate_proj", "out_proj"):
            setattr(self, name, getattr(self, name).to(dtype))

    def forward(self, h: torch.Tensor, batch, cache, layer: int, state: MatrixMemoryState) -> D.SublayerTerms:
        """The sublayer's output for input ``h``; ``layer``: the attention's place in the cache; carries ``state`` on."""
        a, m, at = self.attn, self.memory, self.offsets
        packed = F.linear_rows(h, self.in_proj)
        z = D.few_outputs(h, self.gate_proj)
        D.qkv_head_finish(packed, cache, layer, batch, heads=a.heads, dim=a.padded_dim, q_off=at["left.q"], k_off=at["left.k"], v_off=at["left.v"],
                          q_weight=self.ones, k_weight=self.ones, true_dim=a.dim, eps=self.eps)
        heads = torch.empty((h.shape[0], self.left_width + self.right_width), device=h.device, dtype=h.dtype)
        q = packed[:, at["left.q"]:at["left.k"]].unflatten(1, (a.heads, a.padded_dim))
        cache.attend(layer, q, batch, a.scale, out=heads[:, :self.left_width].unflatten(1, (a.heads, a.padded_vdim)), chunk=a.chunk,
                     slopes=self.slopes, out_scale=self.left_scale)
        D.matrix_memory(packed[:, at["right.q"]:at["right.k"]], packed[:, at["right.k"]:at["right.v"]], packed[:, at["right.v"]:at["right.g"]],
                        packed[:, at["right.g"]:], z, self.i_bias, self.f_bias, self.norm, state, batch, heads[:, self.left_width:], heads=m.heads,
                        dim=m.dim, vdim=m.vdim, cap=m.gate_cap, eps=self.eps, out_scale=self.right_scale)
        return D.SublayerTerms(dense=F.linear_rows(heads, self.out_proj))

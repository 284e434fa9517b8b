"""Zolorax: a pre-norm decoder that mixes windowed attention, real-gated linear recurrences, dense and routed feed-forwards.

Every layer adds ``mixer(norm1(x))`` and then ``ff(norm2(x))`` to the fp32 residual stream
(:class:`~ferrotorch_b200.nn.gated_attention.ResidualRMSNorm`, weights stored around zero).  Mixers: attention with per-head
query / key norm, YaRN-scaled rotation of part of a head, a sliding window, a sink per head and an output gate per element,
over keys and values of its own or of an earlier layer (:class:`~ferrotorch_b200.nn.gated_attention.GatedAttention`); or a
recurrent block (:class:`~ferrotorch_b200.nn.recurrent.RGLRUBlock`).  Feed-forwards: squared ReLU, routed experts, or none
(:mod:`~ferrotorch_b200.nn.feed_forward`).  Layers may differ in every size and come in any order.  The model runs over a
paged KV cache with recurrent states only (:class:`~ferrotorch_b200.models.serving.PagedStepper`, ``ContinuousBatcher``,
``generation.generate``)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.feed_forward import ExpertSpec, PackedMLP, RoutedExperts
from ..nn.gated_attention import GatedAttention, ResidualRMSNorm
from ..nn.packed_block import AttentionSpec, RotarySpec, YarnScaling, pad_to, round_up
from ..nn.paged import PagedKVCache, PagedSession, RaggedBatch
from ..nn.recurrent import RGLRUBlock, RGLRUSpec, RGLRUState
from ..ops import functional as F

ARCHITECTURE = "Zolorax"


@dataclass
class ZoloraxLayerConfig:
    mixer: AttentionSpec | RGLRUSpec
    mlp: int | ExpertSpec | None = None           # width of a dense feed-forward, experts, or none

    @property
    def is_attention(self) -> bool:
        return isinstance(self.mixer, AttentionSpec)


def _read_rotary(rot: dict | None) -> RotarySpec | None:
    if not rot:
        return None
    s = rot.get("scaling")
    return RotarySpec(int(rot["dims"]), float(rot["base"]),
                      YarnScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None)


def _write_rotary(rot: RotarySpec) -> dict:
    out = {"dims": rot.dims, "base": rot.base}
    if rot.scaling is not None:
        out["scaling"] = dict(vars(rot.scaling))
    return out


@dataclass
class ZoloraxConfig:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)            # of ZoloraxLayerConfig
    norm_eps: float = 1e-6
    max_position_embeddings: int | None = None            # nothing in the model limits positions

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def pattern(cls, vocab_size: int, hidden_size: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, experts: int = 8,
                top: int = 2, window: int = 1024, width: int | None = None, blocks: int | None = None, conv: int = 4,
                **kw) -> "ZoloraxConfig":
        """Layers in groups of six: recurrent, recurrent, attention, attention over the keys of the layer before it, recurrent,
        recurrent; dense and routed feed-forwards (``top`` experts of width ``ff / top``) in turn.  ``experts`` 0: all dense."""
        width = width or hidden_size
        rotary = RotarySpec(dim // 2, 10000.0, YarnScaling(4.0, 4096.0))
        layers = []
        for i in range(n_layers):
            if i % 6 in (2, 3):
                mixer = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window=window, rotary=rotary, kv_from=i - 1 if i % 6 == 3 else None)
            else:
                mixer = RGLRUSpec(width, blocks or heads, conv)
            layers.append(ZoloraxLayerConfig(mixer, ExpertSpec(experts, top, ff // top) if experts and i % 2 else ff))
        out = cls(vocab_size, hidden_size, layers, **kw)
        out.validate()
        return out

    @classmethod
    def preset_3b(cls) -> "ZoloraxConfig":
        """Layer sizes of a model that reads about three billion of its parameters per token (no trained weights exist)."""
        return cls.pattern(128256, 3072, 24, 24, 8, 128, 8192, experts=8, top=2, window=2048)

    @classmethod
    def tiny(cls) -> "ZoloraxConfig":
        """A few layers for smoke tests."""
        return cls.pattern(1000, 128, 6, 4, 2, 32, 192, experts=4, top=2, window=40)

    @classmethod
    def from_dict(cls, cfg: dict | str) -> "ZoloraxConfig":
        """Build from a ``config.json`` dict or path."""
        if isinstance(cfg, str):
            with open(cfg) as f:
                cfg = json.load(f)
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError("ZoloraxConfig: architecture is %r" % (cfg.get("architecture"),))
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry.get("type") == "attention":
                mask, source = m.get("mask"), m.get("kv_from")
                mixer = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                      window=int(mask["size"]) if mask else None, rotary=_read_rotary(m.get("rot")),
                                      kv_from=int(source) if source is not None else None)
            elif entry.get("type") == "rglru":
                mixer = RGLRUSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
            else:
                raise ValueError("ZoloraxConfig: layer %d has unknown mixer type %r" % (i, entry.get("type")))
            if mlp is None:
                ff = None
            elif mlp.get("kind") == "dense":
                ff = int(mlp["ff"])
            elif mlp.get("kind") == "moe":
                ff = ExpertSpec(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]))
            else:
                raise ValueError("ZoloraxConfig: layer %d has unknown feed-forward kind %r" % (i, mlp.get("kind")))
            layers.append(ZoloraxLayerConfig(mixer, ff))
        out = cls(int(cfg["vocab"]), int(cfg["width"]), layers, float(cfg["norm"]["eps"]))
        out.validate()
        return out

    def to_dict(self) -> dict:
        layers = []
        for s in self.layers:
            a = s.mixer
            if s.is_attention:
                mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.window is not None:
                    mixer["mask"] = {"size": a.window}
                if a.rotary is not None:
                    mixer["rot"] = _write_rotary(a.rotary)
                if a.kv_from is not None:
                    mixer["kv_from"] = a.kv_from
            else:
                mixer = {"width": a.width, "blocks": a.blocks, "conv": a.conv}
            mlp = s.mlp
            if isinstance(mlp, ExpertSpec):
                mlp = {"kind": "moe", "router": {"experts": mlp.experts, "top": mlp.top}, "expert": {"ff": mlp.ff}}
            elif mlp is not None:
                mlp = {"kind": "dense", "ff": mlp}
            layers.append({"type": "attention" if s.is_attention else "rglru", "mixer": mixer, "mlp": mlp})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "layers": layers}

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers)) < 1:
            raise ValueError("ZoloraxConfig: vocabulary, width and layers must be positive")
        for i, s in enumerate(self.layers):
            s.mixer.validate()
            if isinstance(s.mlp, ExpertSpec):
                s.mlp.validate()
            elif s.mlp is not None and s.mlp < 1:
                raise ValueError("ZoloraxConfig: layer %d: ff must be positive or absent" % i)
            j = s.mixer.kv_from if s.is_attention else None
            if j is not None:
                if not 0 <= j < i or not self.layers[j].is_attention or self.layers[j].mixer.kv_from is not None:
                    raise ValueError("ZoloraxConfig: layer %d reads the keys of layer %d, which has none ahead of it" % (i, j))
                a, b = s.mixer, self.layers[j].mixer
                if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                    raise ValueError("ZoloraxConfig: layers %d and %d share keys of different sizes" % (j, i))

    def num_parameters(self) -> int:
        W = self.hidden_size
        total = 2 * self.vocab_size * W + W
        for s in self.layers:
            m = s.mixer
            total += W * (1 if s.mlp is None else 2)
            if s.is_attention:
                total += W * m.heads * (m.dim + 2 * m.vdim) + m.dim + m.heads
                if m.kv_from is None:
                    total += W * m.kv_heads * (m.dim + m.vdim) + m.dim
            else:
                total += 3 * W * m.width + m.width * (m.conv + 2 * m.block + 6)
            if isinstance(s.mlp, ExpertSpec):
                total += s.mlp.experts * W * (1 + 3 * s.mlp.ff)
            elif s.mlp is not None:
                total += 2 * W * s.mlp
        return total


class ZoloraxLayer(nn.Module):
    def __init__(self, cfg: ZoloraxConfig, spec: ZoloraxLayerConfig):
        super().__init__()
        W = cfg.hidden_size
        self.norm1 = ResidualRMSNorm(W, cfg.norm_eps, offset=1.0)
        self.mixer = GatedAttention(W, spec.mixer, cfg.norm_eps) if spec.is_attention else RGLRUBlock(W, spec.mixer)
        self.norm2 = self.mlp = None
        if spec.mlp is not None:
            self.norm2 = ResidualRMSNorm(W, cfg.norm_eps, offset=1.0)
            self.mlp = RoutedExperts(W, spec.mlp) if isinstance(spec.mlp, ExpertSpec) else PackedMLP(W, spec.mlp)

    def parts(self) -> list:
        """``(prefix of the checkpoint names, module)`` of the sublayers."""
        return [("mix.", self.mixer)] + ([("mlp.", self.mlp)] if self.mlp is not None else [])

    def norms(self) -> list:
        return [("norm1", self.norm1)] + ([("norm2", self.norm2)] if self.norm2 is not None else [])


class ZoloraxForCausalLM(nn.Module):
    """Weights are buffers (inference only).  ``dtype`` of the matrices: bf16 (served) or fp32 (everything in 32-bit); norms,
    the residual stream, the recurrence and routing are fp32 in both."""

    def __init__(self, cfg: ZoloraxConfig, dtype: torch.dtype = torch.bfloat16, device="cpu"):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("ZoloraxForCausalLM: dtype must be bfloat16 or float32")
        self.config, self.dtype = cfg, dtype
        width = round_up(cfg.hidden_size, 8)
        # where a layer's keys and values lie in the cache: layers that read another's share its place
        places: dict = {}
        for i, s in enumerate(cfg.layers):
            if s.is_attention:
                places[i] = len(set(places.values())) if s.mixer.kv_from is None else places[s.mixer.kv_from]
        self._places = places
        with torch.device(device):
            self.layers = nn.ModuleList()
            for s in cfg.layers:
                layer = ZoloraxLayer(cfg, s)
                for _, part in layer.parts():
                    part.cast_(dtype)
                self.layers.append(layer)
            self.final_norm = ResidualRMSNorm(cfg.hidden_size, cfg.norm_eps, offset=1.0)
            self.register_buffer("embed", torch.zeros(cfg.vocab_size, width, dtype=dtype))
            self.register_buffer("head", torch.zeros(round_up(cfg.vocab_size, 8), width, dtype=dtype))

    # ------------------------------------------------------------------ weights
    def load_tensors(self, sd: dict) -> None:
        """Load the checkpoint's tensors (names ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
        ``final.norm``, ``head``); every tensor must be used and have its shape."""
        left, c = dict(sd), self.config

        def take(name):
            if name not in left:
                raise KeyError("checkpoint has no tensor %r" % name)
            return left.pop(name)

        for name, buf in (("embed", self.embed), ("head", self.head)):
            t = take(name)
            if tuple(t.shape) != (c.vocab_size, c.hidden_size):
                raise ValueError("%s must have shape %s, got %s" % (name, (c.vocab_size, c.hidden_size), tuple(t.shape)))
            buf.copy_(pad_to(t, *buf.shape))
        self.final_norm.load(take("final.norm"))
        for i, layer in enumerate(self.layers):
            pre = "l%d." % i
            for name, norm in layer.norms():
                norm.load(take(pre + name))
            for part, module in layer.parts():
                module.load({n: take(pre + part + n) for n in module.tensor_names()})
        if left:
            raise KeyError("checkpoint has tensors this model does not know: %s" % sorted(left)[:8])

    def random_(self, std: float = 0.02, seed: int = 0) -> "ZoloraxForCausalLM":
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        c = self.config
        for buf in (self.embed, self.head):
            buf[:c.vocab_size, :c.hidden_size].copy_(torch.randn(c.vocab_size, c.hidden_size, device=buf.device, generator=g) * std)
        for layer in self.layers:
            for _, part in layer.parts():
                part.random_(std, g)
        return self

    @classmethod
    def tiny_random(cls, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "ZoloraxForCausalLM":
        return cls(ZoloraxConfig.tiny(), dtype, device).random_()

    def checkpoint_tensors(self) -> dict:
        """The weights under their checkpoint names, in their true sizes."""
        c = self.config
        out = {"embed": self.embed[:, :c.hidden_size], "head": self.head[:c.vocab_size, :c.hidden_size], "final.norm": self.final_norm.unpack()}
        for i, layer in enumerate(self.layers):
            pre = "l%d." % i
            out.update({pre + name: norm.unpack() for name, norm in layer.norms()})
            for part, module in layer.parts():
                out.update({pre + part + n: t for n, t in module.unpack().items()})
        return {k: v.contiguous() for k, v in out.items()}

    def save_pretrained(self, path: str) -> None:
        """Write ``config.json`` and ``model.safetensors``."""
        from ..serialize.state import save_safetensors

        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.config.to_dict(), f, indent=1)
        save_safetensors(self.checkpoint_tensors(), os.path.join(path, "model.safetensors"))

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "ZoloraxForCausalLM":
        """The model of a directory with ``config.json`` and ``model.safetensors`` (or shards with an index)."""
        from ..serialize.state import load_safetensors_auto

        model = cls(ZoloraxConfig.from_dict(os.path.join(path, "config.json")), dtype, device)
        model.load_tensors(load_safetensors_auto(path))
        return model

    # ------------------------------------------------------------------ inference over a paged cache
    def make_paged_cache(self, num_blocks: int, block_size: int, max_seqs: int, max_seq_len: int) -> PagedKVCache:
        """Pages for the layers with keys of their own, a state per slot (and one for padding rows) for recurrent layers."""
        layers = self.config.layers
        specs = [s.mixer for s in layers if s.is_attention and s.mixer.kv_from is None]
        cache = PagedKVCache(len(specs), [a.kv_heads for a in specs], [a.padded_dim for a in specs], num_blocks, max_seqs, max_seq_len,
                             block_size, self.embed.device, self.dtype, v_head_dim=[a.padded_vdim for a in specs])
        cache.states = {i: RGLRUState(max_seqs + 1, s.mixer, self.embed.device, self.dtype) for i, s in enumerate(layers) if not s.is_attention}
        return cache

    @torch.no_grad()
    def paged_forward(self, batch: RaggedBatch, cache: PagedKVCache, on_layer=None) -> torch.Tensor:
        """One pass over a ragged batch: fp32 logits ``[wanted rows, vocab]``.  ``on_layer(i, x)`` sees the residual stream
        (padded width) after every layer."""
        x = pending = None                                # pending: experts' outputs that the next norm adds to x
        for i, layer in enumerate(self.layers):
            if x is None:
                x, h = layer.norm1.gather(batch.tokens, self.embed, self.dtype)
            else:
                h = layer.norm1(x, pending=pending, update=pending is not None, out_dtype=self.dtype)
                pending = None
            if i in self._places:
                layer.mixer(x, h, batch, cache, self._places[i])
            else:
                layer.mixer(x, h, batch, cache.states[i])
            if layer.mlp is not None:
                h = layer.norm2(x, out_dtype=self.dtype)
                pending = layer.mlp(h) if isinstance(layer.mlp, RoutedExperts) else layer.mlp(x, h)
            if on_layer is not None:
                on_layer(i, x if pending is None else x + pending[0][pending[1].long()].float().sum(1))
        if batch.n_want == 0:
            return torch.empty((0, self.config.vocab_size), device=x.device)
        h = self.final_norm(x, rows=batch.last, pending=pending, out_dtype=self.dtype)
        return F.linear_f32_out(h, self.head)[:, :self.config.vocab_size]

    # ------------------------------------------------------------------ dense entry points (models.generation)
    def make_caches(self, batch: int, max_len: int, device=None, dtype=None) -> PagedSession:
        return PagedSession(self, batch, max_len)

    def forward(self, input_ids: torch.Tensor, *, caches: PagedSession | None = None, last_token_only: bool = False) -> torch.Tensor:
        """Logits ``[B, S, vocab]`` (or ``[B, 1, vocab]``) of equally long sequences, continuing ``caches`` when given."""
        session = caches if caches is not None else PagedSession(self, *input_ids.shape)
        return session.extend(input_ids, last_token_only)

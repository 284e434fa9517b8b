"""Tenalorn: a decoder whose residual is several streams, with attention beside matrix memories, latent attention and routed experts.

The embedding adds a row hashed from the previous and the present token.  Every sublayer reads a weighted sum of the fp32 residual
streams through an RMS norm and leaves its output in all of them (:class:`~ferrotorch_b200.nn.streams.StreamMixing`).  Mixers:
chunked attention with a distance bias beside matrix memories with exponential gates
(:class:`~ferrotorch_b200.nn.parallel_mixer.AttentionMemoryMixer`), or latent attention
(:class:`~ferrotorch_b200.nn.latent_attention.LatentAttention`).  Feed-forwards: routed experts with identity experts and a shared
one (:class:`~ferrotorch_b200.nn.feed_forward.RoutedExperts`), or none.  Logits are capped softly.  Layers may differ in every
size and come in any order.  The model runs over a paged KV cache with recurrent states only
(:class:`~ferrotorch_b200.models.serving.PagedStepper`, ``ContinuousBatcher``, ``generation.generate``)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.feed_forward import ExpertSpec, RoutedExperts
from ..nn.gated_attention import ResidualRMSNorm
from ..nn.latent_attention import LatentAttention, LatentSpec
from ..nn.packed_block import AttentionSpec, RotarySpec, pad_to, round_up
from ..nn.paged import PagedKVCache, PagedSession, RaggedBatch
from ..nn.parallel_mixer import AttentionMemoryMixer
from ..nn.recurrent import MatrixMemorySpec, MatrixMemoryState
from ..nn.streams import StreamMixing
from ..ops import decoder as D
from ..ops import functional as F

ARCHITECTURE = "Tenalorn"


@dataclass
class ParallelSpec:
    """Attention and matrix memories side by side, weighted by two constants."""
    left: AttentionSpec
    right: MatrixMemorySpec
    left_scale: float = 1.0
    right_scale: float = 1.0

    def validate(self) -> None:
        self.left.validate()
        self.right.validate()


@dataclass
class TenalornLayerConfig:
    mixer: ParallelSpec | LatentSpec
    mlp: ExpertSpec | None = None

    @property
    def is_parallel(self) -> bool:
        return isinstance(self.mixer, ParallelSpec)


@dataclass
class BigramSpec:
    """Table of token pairs: row ``(previous * mul_prev + token * mul_cur) mod buckets``, row ``buckets`` for a first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class TenalornConfig:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)            # of TenalornLayerConfig
    streams: int = 2
    bigram: BigramSpec = field(default_factory=lambda: BigramSpec(4099, 31, 7))
    embedding_scale: float = 1.0
    logit_softcap: float = 30.0
    norm_eps: float = 1e-5
    max_position_embeddings: int | None = None            # nothing in the model limits positions

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def experts(experts: int, top: int, ff: int, identity: int = 0, shared_ff: int | None = None) -> ExpertSpec:
        """Experts by this design's rules: corrected softmax scores, normalised weights on the outputs."""
        return ExpertSpec(experts, top, ff, score="softmax", correction=True, normalize=True, scale="output", identity=identity, shared_ff=shared_ff)

    @classmethod
    def pattern(cls, vocab_size: int, hidden_size: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, *, chunk: int = 1024,
                memory_heads: int | None = None, memory_dim: int | None = None, memory_vdim: int | None = None, rank: int = 512,
                rot_dim: int | None = None, experts: int = 8, top: int = 2, identity: int = 1, shared_ff: int | None = None, **kw) -> "TenalornConfig":
        """Layers in groups of three: parallel, latent attention, parallel; ``top`` of ``experts`` (and ``identity``) of width ``ff``."""
        rot = rot_dim or max(2, dim // 4)
        layers = []
        for i in range(n_layers):
            if i % 3 == 1:
                mixer = LatentSpec(heads, dim - rot, rot, dim, rank, dim ** -0.5, RotarySpec(rot, 10000.0, interleaved=True))
            else:
                mixer = ParallelSpec(AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, chunk=chunk, distance_bias=True),
                                     MatrixMemorySpec(memory_heads or max(1, heads // 2), memory_dim or dim, memory_vdim or dim, 15.0))
            layers.append(TenalornLayerConfig(mixer, cls.experts(experts, top, ff, identity, shared_ff or ff)))
        out = cls(vocab_size, hidden_size, layers, **kw)
        out.validate()
        return out

    @classmethod
    def preset_3b(cls) -> "TenalornConfig":
        """Layer sizes of a model that reads about three billion of its parameters per token (no trained weights exist)."""
        return cls.pattern(128256, 3072, 24, 24, 8, 128, 2816, chunk=2048, memory_heads=12, memory_dim=128, memory_vdim=128, bigram=BigramSpec(131071, 1031, 17))

    @classmethod
    def tiny(cls) -> "TenalornConfig":
        """A few layers for smoke tests."""
        return cls.pattern(1000, 128, 3, 4, 2, 32, 64, chunk=40, rank=48, memory_heads=2, experts=4, bigram=BigramSpec(509, 29, 3))

    @classmethod
    def from_dict(cls, cfg: dict | str) -> "TenalornConfig":
        """Build from a ``config.json`` dict or path."""
        if isinstance(cfg, str):
            with open(cfg) as f:
                cfg = json.load(f)
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError("TenalornConfig: architecture is %r" % (cfg.get("architecture"),))
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry.get("type") == "parallel":
                a, b = m["left"], m["right"]
                mask = a.get("mask")
                mixer = ParallelSpec(AttentionSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                                                   chunk=int(mask["size"]) if mask else None, distance_bias=True),
                                     MatrixMemorySpec(int(b["heads"]), int(b["dim"]), int(b["vdim"]), float(b["gate_cap"])),
                                     float(m["left_scale"]), float(m["right_scale"]))
            elif entry.get("type") == "latent_attention":
                rot = m["rot"]
                mixer = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                                   RotarySpec(int(rot["dims"]), float(rot["base"]), interleaved=True))
            else:
                raise ValueError("TenalornConfig: layer %d has unknown mixer type %r" % (i, entry.get("type")))
            if mlp is None:
                ff = None
            elif mlp.get("kind") == "moe":
                r, shared = mlp["router"], mlp.get("shared")
                ff = cls.experts(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(r.get("identity") or 0),
                                 int(shared["ff"]) if shared else None)
            else:
                raise ValueError("TenalornConfig: layer %d has unknown feed-forward kind %r" % (i, mlp.get("kind")))
            layers.append(TenalornLayerConfig(mixer, ff))
        emb = cfg["embedding"]
        big = emb["bigram"]
        out = cls(int(cfg["vocab"]), int(cfg["width"]), layers, int(cfg["streams"]), BigramSpec(int(big["buckets"]), int(big["mul_prev"]), int(big["mul_cur"])),
                  float(emb["scale"]), float(cfg["logit_softcap"]), float(cfg["norm"]["eps"]))
        out.validate()
        return out

    def to_dict(self) -> dict:
        layers = []
        for s in self.layers:
            if s.is_parallel:
                a, b = s.mixer.left, s.mixer.right
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.chunk is not None:
                    left["mask"] = {"size": a.chunk}
                mixer = {"left": left, "right": {"heads": b.heads, "dim": b.dim, "vdim": b.vdim, "gate_cap": b.gate_cap},
                         "left_scale": s.mixer.left_scale, "right_scale": s.mixer.right_scale}
            else:
                a = s.mixer
                mixer = {"heads": a.heads, "dim": a.dim, "rot_dim": a.rot_dim, "vdim": a.vdim, "kv_rank": a.rank, "scale": a.scale,
                         "rot": {"base": a.rotary.base, "dims": a.rotary.dims}}
            mlp = None
            if s.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": s.mlp.ff}, "router": {"experts": s.mlp.experts, "identity": s.mlp.identity, "top": s.mlp.top}}
                if s.mlp.shared_ff is not None:
                    mlp["shared"] = {"ff": s.mlp.shared_ff}
            layers.append({"type": "parallel" if s.is_parallel else "latent_attention", "mixer": mixer, "mlp": mlp})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                "embedding": {"scale": self.embedding_scale, "bigram": {"buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur}},
                "norm": {"eps": self.norm_eps}, "logit_softcap": self.logit_softcap, "layers": layers}

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers), self.bigram.buckets) < 1:
            raise ValueError("TenalornConfig: vocabulary, width, layers and buckets must be positive")
        if not 1 <= self.streams <= 16:
            raise ValueError("TenalornConfig: %d streams (1 to 16)" % self.streams)
        if not self.logit_softcap > 0:
            raise ValueError("TenalornConfig: logit_softcap must be positive")
        for s in self.layers:
            s.mixer.validate()
            if s.mlp is not None:
                s.mlp.validate()

    def num_parameters(self) -> int:
        W, hc = self.hidden_size, self.streams * (self.streams + 2)
        total = (2 * self.vocab_size + self.bigram.buckets + 1) * W + W
        for s in self.layers:
            total += (W + hc) * (1 if s.mlp is None else 2)
            if s.is_parallel:
                a, b = s.mixer.left, s.mixer.right
                total += W * (a.heads + a.kv_heads) * (a.dim + a.vdim)
                total += W * b.heads * (2 * b.dim + 3 * b.vdim + 2) + b.heads * (b.vdim + 2)
            else:
                a = s.mixer
                total += W * (a.heads * (a.dim + a.rot_dim + 2 * a.vdim) + a.rank + a.rot_dim) + a.rank * (1 + a.heads * (a.dim + a.vdim))
            if s.mlp is not None:
                total += s.mlp.outputs * (W + 1) + 3 * W * (s.mlp.experts * s.mlp.ff + (s.mlp.shared_ff or 0))
        return total


class TenalornLayer(nn.Module):
    def __init__(self, cfg: TenalornConfig, spec: TenalornLayerConfig):
        super().__init__()
        W, m = cfg.hidden_size, spec.mixer
        self.norm1, self.hc1 = ResidualRMSNorm(W, cfg.norm_eps), StreamMixing(cfg.streams)
        if spec.is_parallel:
            self.mixer = AttentionMemoryMixer(W, m.left, m.right, m.left_scale, m.right_scale, cfg.norm_eps)
        else:
            self.mixer = LatentAttention(W, m, cfg.norm_eps)
        self.norm2 = self.hc2 = self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.hc2 = ResidualRMSNorm(W, cfg.norm_eps), StreamMixing(cfg.streams)
            self.mlp = RoutedExperts(W, spec.mlp)

    def parts(self) -> list:
        """``(prefix of the checkpoint names, module)`` of what has several tensors."""
        out = [("mix.", self.mixer), ("hc1.", self.hc1)]
        return out + ([("mlp.", self.mlp), ("hc2.", self.hc2)] if self.mlp is not None else [])

    def norms(self) -> list:
        return [("norm1", self.norm1)] + ([("norm2", self.norm2)] if self.norm2 is not None else [])


class TenalornForCausalLM(nn.Module):
    """Weights are buffers (inference only).  ``dtype`` of the matrices: bf16 (served) or fp32 (everything in 32-bit); norms,
    the residual streams, gates and states of the memories and routing are fp32 in both."""

    def __init__(self, cfg: TenalornConfig, dtype: torch.dtype = torch.bfloat16, device="cpu"):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("TenalornForCausalLM: dtype must be bfloat16 or float32")
        self.config, self.dtype = cfg, dtype
        width = round_up(cfg.hidden_size, 8)
        with torch.device(device):
            self.layers = nn.ModuleList()
            for s in cfg.layers:
                layer = TenalornLayer(cfg, s)
                for part in (layer.mixer, layer.mlp):
                    if part is not None:
                        part.cast_(dtype)
                self.layers.append(layer)
            self.final_norm = ResidualRMSNorm(cfg.hidden_size, cfg.norm_eps)
            self.register_buffer("embed", torch.zeros(cfg.vocab_size, width, dtype=dtype))
            self.register_buffer("bigram", torch.zeros(cfg.bigram.buckets + 1, width, dtype=dtype))
            self.register_buffer("head", torch.zeros(round_up(cfg.vocab_size, 8), width, dtype=dtype))
            self.register_buffer("sum_of_streams", torch.ones(cfg.streams))

    # ------------------------------------------------------------------ weights
    def _tables(self) -> list:
        c = self.config
        return [("embed", self.embed, c.vocab_size), ("bigram", self.bigram, c.bigram.buckets + 1), ("head", self.head, c.vocab_size)]

    def load_tensors(self, sd: dict) -> None:
        """Load the checkpoint's tensors (names ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.hc1.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ..,
        ``final.norm``, ``head``); every tensor must be used and have its shape."""
        left, c = dict(sd), self.config

        def take(name):
            if name not in left:
                raise KeyError("checkpoint has no tensor %r" % name)
            return left.pop(name)

        for name, buf, rows in self._tables():
            t = take(name)
            if tuple(t.shape) != (rows, c.hidden_size):
                raise ValueError("%s must have shape %s, got %s" % (name, (rows, c.hidden_size), tuple(t.shape)))
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

    def random_(self, std: float = 0.02, seed: int = 0) -> "TenalornForCausalLM":
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        c = self.config
        for _, buf, rows in self._tables():
            buf[:rows, :c.hidden_size].copy_(torch.randn(rows, c.hidden_size, device=buf.device, generator=g) * std)
        for layer in self.layers:
            for _, part in layer.parts():
                part.random_(std, g)
        return self

    @classmethod
    def tiny_random(cls, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "TenalornForCausalLM":
        return cls(TenalornConfig.tiny(), dtype, device).random_()

    def checkpoint_tensors(self) -> dict:
        """The weights under their checkpoint names, in their true sizes."""
        c = self.config
        out = {name: buf[:rows, :c.hidden_size] for name, buf, rows in self._tables()}
        out["final.norm"] = self.final_norm.unpack()
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
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "TenalornForCausalLM":
        """The model of a directory with ``config.json`` and ``model.safetensors`` (or shards with an index)."""
        from ..serialize.state import load_safetensors_auto

        model = cls(TenalornConfig.from_dict(os.path.join(path, "config.json")), dtype, device)
        model.load_tensors(load_safetensors_auto(path))
        return model

    # ------------------------------------------------------------------ inference over a paged cache
    def make_paged_cache(self, num_blocks: int, block_size: int, max_seqs: int, max_seq_len: int) -> PagedKVCache:
        """Pages for keys and values or latents of every layer and for the tokens, a state per slot (and one for padding rows)
        for matrix memories."""
        layers, dev = self.config.layers, self.embed.device
        shapes = [(s.mixer.left.kv_heads, s.mixer.left.padded_dim, s.mixer.left.padded_vdim) if s.is_parallel
                  else (1, s.mixer.row_size, s.mixer.padded_rank) for s in layers]
        heads, dims, vdims = (list(t) for t in zip(*shapes))
        cache = PagedKVCache(len(layers), heads, dims, num_blocks, max_seqs, max_seq_len, block_size, dev, self.dtype, v_head_dim=vdims,
                             values_in_keys=[not s.is_parallel for s in layers])
        cache.keep_tokens()
        cache.states = {i: MatrixMemoryState(max_seqs + 1, s.mixer.right, dev) for i, s in enumerate(layers) if s.is_parallel}
        return cache

    @torch.no_grad()
    def paged_forward(self, batch: RaggedBatch, cache: PagedKVCache, on_layer=None) -> torch.Tensor:
        """One pass over a ragged batch: fp32 logits ``[wanted rows, vocab]``.  ``on_layer(i, x)`` sees the sum of the residual
        streams (padded width) after every layer."""
        c, first = self.config, self.layers[0]
        x, h = D.embed_bigram(batch, cache, self.embed, self.bigram, c.embedding_scale, c.bigram.mul_prev, c.bigram.mul_cur, first.hc1.into,
                              first.norm1.weight, c.norm_eps, count=c.hidden_size, out_dtype=self.dtype)
        x = x[:, None].expand(-1, c.streams, -1)          # all streams are equal until the first sublayer
        last = len(self.layers) - 1
        for i, layer in enumerate(self.layers):
            y = layer.mixer(h, batch, cache, i, cache.states[i]) if i in cache.states else layer.mixer(h, batch, cache, i)
            ends = layer.hc1
            if layer.mlp is not None:
                x, h = layer.hc1.step(x, y, layer.hc2.into, layer.norm2, self.dtype)
                y, ends = layer.mlp(h), layer.hc2
            if on_layer is not None:
                on_layer(i, torch.einsum("nsh,s->nh", x, ends.mix.sum(1)) + ends.out.sum() * y.total())
            if i < last:
                after = self.layers[i + 1]
                x, h = ends.step(x, y, after.hc1.into, after.norm1, self.dtype)
            elif batch.n_want:
                _, h = ends.step(x, y, self.sum_of_streams, self.final_norm, self.dtype, rows=batch.last)
        if batch.n_want == 0:
            return torch.empty((0, c.vocab_size), device=x.device)
        return D.softcap_(F.linear_f32_out(h, self.head), c.logit_softcap)[:, :c.vocab_size]

    # ------------------------------------------------------------------ dense entry points (models.generation)
    def make_caches(self, batch: int, max_len: int, device=None, dtype=None) -> PagedSession:
        return PagedSession(self, batch, max_len)

    def forward(self, input_ids: torch.Tensor, *, caches: PagedSession | None = None, last_token_only: bool = False) -> torch.Tensor:
        """Logits ``[B, S, vocab]`` (or ``[B, 1, vocab]``) of equally long sequences, continuing ``caches`` when given."""
        session = caches if caches is not None else PagedSession(self, *input_ids.shape)
        return session.extend(input_ids, last_token_only)

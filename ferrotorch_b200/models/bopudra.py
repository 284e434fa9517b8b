"""Bopudra: a decoder with parallel sublayers, dynamic-tanh norms and position-free attention.

Every layer computes ``h = norm(x)`` once (:class:`~ferrotorch_b200.nn.packed_block.DynamicTanh`) and adds attention and
feed-forward of the same ``h`` to the fp32 residual stream.  Attention: grouped heads whose key and value sizes may
differ, RMS norm over the whole query and key projections, no rotation, a query temperature that grows with the
logarithm of the position, one sigmoid output gate per head.  Feed-forward: ``W_down gelu(W_up h)``, or none.  Layers
may differ in every size.  The model runs over a paged KV cache only
(:class:`~ferrotorch_b200.models.serving.PagedStepper`, ``ContinuousBatcher``, ``generation.generate``)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.packed_block import AttentionSpec, DynamicTanh, PackedParallelBlock, pad_to, round_up
from ..nn.paged import PagedKVCache, PagedSession, RaggedBatch
from ..ops import functional as F

ARCHITECTURE = "Bopudra"


@dataclass
class BopudraLayerConfig:
    attention: AttentionSpec
    ff: int | None = None


@dataclass
class BopudraConfig:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)            # of BopudraLayerConfig
    norm_eps: float = 1e-5
    logit_scale: float = 1.0
    max_position_embeddings: int | None = None            # nothing in the model limits positions

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def uniform(cls, vocab_size: int, hidden_size: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int | None,
                vdim: int | None = None, **kw) -> "BopudraConfig":
        """Equal layers, scores scaled by ``dim ** -0.5``."""
        spec = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, scale=dim ** -0.5, temp_coef=0.1, temp_every=8192)
        out = cls(vocab_size, hidden_size, [BopudraLayerConfig(AttentionSpec(**spec), ff) for _ in range(n_layers)], **kw)
        out.validate()
        return out

    @classmethod
    def preset_8b(cls) -> "BopudraConfig":
        """Layer sizes of an 8-billion-parameter decoder (no trained weights exist)."""
        return cls.uniform(128256, 4096, 32, 32, 8, 128, 21504)

    @classmethod
    def tiny(cls) -> "BopudraConfig":
        """A few layers for smoke tests."""
        return cls.uniform(1000, 128, 3, 4, 1, 32, 352, vdim=48)

    @classmethod
    def from_dict(cls, cfg: dict | str) -> "BopudraConfig":
        """Build from a ``config.json`` dict or path."""
        if isinstance(cfg, str):
            with open(cfg) as f:
                cfg = json.load(f)
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError("BopudraConfig: architecture is %r" % (cfg.get("architecture"),))
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            if entry.get("type") != "attention":
                raise ValueError("BopudraConfig: layer %d has unknown mixer type %r" % (i, entry.get("type")))
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError("BopudraConfig: layer %d has unknown feed-forward kind %r" % (i, mlp.get("kind")))
            temp = m.get("q_temp") or {"coef": 0.0, "every": 1}
            layers.append(BopudraLayerConfig(AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                                           float(temp["coef"]), float(temp["every"])),
                                             int(mlp["ff"]) if mlp is not None else None))
        out = cls(int(cfg["vocab"]), int(cfg["width"]), layers, float(cfg["norm"]["eps"]), float(cfg["logit_scale"]))
        out.validate()
        return out

    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "logit_scale": self.logit_scale,
                "norm": {"eps": self.norm_eps},
                "layers": [{"type": "attention",
                            "mixer": {"heads": s.attention.heads, "kv_heads": s.attention.kv_heads, "dim": s.attention.dim, "vdim": s.attention.vdim,
                                      "scale": s.attention.scale, "q_temp": {"coef": s.attention.temp_coef, "every": s.attention.temp_every}},
                            "mlp": {"kind": "dense", "ff": s.ff} if s.ff else None} for s in self.layers]}

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers)) < 1:
            raise ValueError("BopudraConfig: vocabulary, width and layers must be positive")
        for s in self.layers:
            s.attention.validate()
            if s.ff is not None and s.ff < 1:
                raise ValueError("BopudraConfig: ff must be positive or absent")

    def num_parameters(self) -> int:
        W, total = self.hidden_size, 2 * self.vocab_size * self.hidden_size + 2 * self.hidden_size + 1
        for s in self.layers:
            a = s.attention
            q, k = a.heads * a.dim, a.kv_heads * a.dim
            total += W * (q + k + a.kv_heads * a.vdim + a.heads + a.heads * a.vdim + 2 * (s.ff or 0)) + q + k + 2 * W + 1
        return total


class BopudraForCausalLM(nn.Module):
    """Weights are buffers (inference only).  ``dtype`` of the matrices: bf16 (served) or fp32 (everything in 32-bit);
    norms and the residual stream are fp32 in both."""

    def __init__(self, cfg: BopudraConfig, dtype: torch.dtype = torch.bfloat16, device="cpu"):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("BopudraForCausalLM: dtype must be bfloat16 or float32")
        self.config, self.dtype = cfg, dtype
        width = round_up(cfg.hidden_size, 8)
        with torch.device(device):
            self.norms = nn.ModuleList(DynamicTanh(cfg.hidden_size) for _ in cfg.layers)
            self.blocks = nn.ModuleList()
            for s in cfg.layers:
                block = PackedParallelBlock(cfg.hidden_size, s.attention, s.ff, "gelu", cfg.norm_eps)
                block.cast_(dtype)
                self.blocks.append(block)
            self.final_norm = DynamicTanh(cfg.hidden_size)
            self.register_buffer("embed", torch.zeros(cfg.vocab_size, width, dtype=dtype))
            self.register_buffer("head", torch.zeros(round_up(cfg.vocab_size, 8), width, dtype=dtype))

    # ------------------------------------------------------------------ weights
    def load_tensors(self, sd: dict) -> None:
        """Load the checkpoint's tensors (names ``embed``, ``l<i>.norm1[.alpha|.b]``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
        ``final.norm*``, ``head``); every tensor must be used and have its shape."""
        left = dict(sd)

        def take(name):
            if name not in left:
                raise KeyError("checkpoint has no tensor %r" % name)
            return left.pop(name)

        def norm(module, name):
            module.load(take(name + ".alpha"), take(name), take(name + ".b"))

        c = self.config
        for name, buf in (("embed", self.embed), ("head", self.head)):
            t = take(name)
            if tuple(t.shape) != (c.vocab_size, c.hidden_size):
                raise ValueError("%s must have shape %s, got %s" % (name, (c.vocab_size, c.hidden_size), tuple(t.shape)))
            buf.copy_(pad_to(t, *buf.shape))
        norm(self.final_norm, "final.norm")
        for i, (n, block) in enumerate(zip(self.norms, self.blocks)):
            pre = "l%d." % i
            norm(n, pre + "norm1")
            mix = {k: take(pre + "mix." + k) for k in ("q", "k", "v", "o", "g", "q.norm", "k.norm")}
            up, down = (take(pre + "mlp.up"), take(pre + "mlp.down")) if block.ff else (None, None)
            block.load(mix["q"], mix["k"], mix["v"], mix["o"], up, down, mix["g"], mix["q.norm"], mix["k.norm"])
        if left:
            raise KeyError("checkpoint has tensors this model does not know: %s" % sorted(left)[:8])

    def random_(self, std: float = 0.02, seed: int = 0) -> "BopudraForCausalLM":
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        c = self.config
        for buf in (self.embed, self.head):
            buf[:c.vocab_size, :c.hidden_size].copy_(torch.randn(c.vocab_size, c.hidden_size, device=buf.device, generator=g) * std)
        for block in self.blocks:
            block.random_(std, g)
        return self

    @classmethod
    def tiny_random(cls, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "BopudraForCausalLM":
        return cls(BopudraConfig.tiny(), dtype, device).random_()

    def checkpoint_tensors(self) -> dict:
        """The weights under their checkpoint names, in their true sizes."""
        c = self.config
        out = {"embed": self.embed[:, :c.hidden_size], "head": self.head[:c.vocab_size, :c.hidden_size]}
        named = [("final.norm", self.final_norm)] + [("l%d.norm1" % i, n) for i, n in enumerate(self.norms)]
        for name, n in named:
            out.update({name: n.weight[:c.hidden_size], name + ".b": n.bias[:c.hidden_size], name + ".alpha": n.alpha})
        for i, block in enumerate(self.blocks):
            parts = block.unpack()
            for name, key in (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("g", "gate"), ("q.norm", "q_norm"), ("k.norm", "k_norm")):
                out["l%d.mix.%s" % (i, name)] = parts[key]
            if block.ff:
                out.update({"l%d.mlp.up" % i: parts["up"], "l%d.mlp.down" % i: parts["down"]})
        return {k: v.contiguous() for k, v in out.items()}

    def save_pretrained(self, path: str) -> None:
        """Write ``config.json`` and ``model.safetensors``."""
        from ..serialize.state import save_safetensors

        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.config.to_dict(), f, indent=1)
        save_safetensors(self.checkpoint_tensors(), os.path.join(path, "model.safetensors"))

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "BopudraForCausalLM":
        """The model of a directory with ``config.json`` and ``model.safetensors`` (or shards with an index)."""
        from ..serialize.state import load_safetensors_auto

        model = cls(BopudraConfig.from_dict(os.path.join(path, "config.json")), dtype, device)
        model.load_tensors(load_safetensors_auto(path))
        return model

    # ------------------------------------------------------------------ inference over a paged cache
    def make_paged_cache(self, num_blocks: int, block_size: int, max_seqs: int, max_seq_len: int) -> PagedKVCache:
        specs = [s.attention for s in self.config.layers]
        return PagedKVCache(len(specs), [a.kv_heads for a in specs], [a.padded_dim for a in specs], num_blocks, max_seqs, max_seq_len,
                            block_size, self.embed.device, self.dtype, v_head_dim=[a.padded_vdim for a in specs])

    @torch.no_grad()
    def paged_forward(self, batch: RaggedBatch, cache: PagedKVCache, on_layer=None) -> torch.Tensor:
        """One pass over a ragged batch: fp32 logits ``[wanted rows, vocab]``.  ``on_layer(i, x)`` sees the residual stream
        (padded width) after every layer."""
        n0 = self.norms[0]
        x, h = F.embedding_dynamic_tanh(batch.tokens, self.embed, n0.alpha, n0.weight, n0.bias, out_dtype=self.dtype)
        last = len(self.blocks) - 1
        for i, block in enumerate(self.blocks):
            h = block(x, h, batch, cache, i, self.norms[i + 1].as_epilogue() if i < last else None)
            if on_layer is not None:
                on_layer(i, x)
        if batch.n_want == 0:
            return torch.empty((0, self.config.vocab_size), device=x.device)
        h = self.final_norm(x.index_select(0, batch.last), scale=self.config.logit_scale, out_dtype=self.dtype)
        return F.linear_f32_out(h, self.head)[:, :self.config.vocab_size]

    # ------------------------------------------------------------------ dense entry points (models.generation)
    def make_caches(self, batch: int, max_len: int, device=None, dtype=None) -> PagedSession:
        return PagedSession(self, batch, max_len)

    def forward(self, input_ids: torch.Tensor, *, caches: PagedSession | None = None, last_token_only: bool = False) -> torch.Tensor:
        """Logits ``[B, S, vocab]`` (or ``[B, 1, vocab]``) of equally long sequences, continuing ``caches`` when given."""
        session = caches if caches is not None else PagedSession(self, *input_ids.shape)
        return session.extend(input_ids, last_token_only)

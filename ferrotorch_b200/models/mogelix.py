"""Mogelix: a post-norm decoder that mixes state-space heads, windowed attention with pooled blocks, dense and routed feed-forwards.

Every sublayer reads the residual itself, and ``x <- norm(alpha x + sigmoid(W x + b) * sublayer(x))``: the sum, its gate and the norm are
one kernel (:func:`~ferrotorch_b200.ops.decoder.sum_norm`), the gate's product rides along in the sublayer's own.  Mixers: state-space
duality (:class:`~ferrotorch_b200.nn.recurrent.StateSpaceBlock`), or attention over a window and the means of the blocks ahead of it, with
rotation scaled by wavelength, RMS norm per head and a sink per head, over keys and values of its own or of an earlier layer
(:class:`~ferrotorch_b200.nn.gated_attention.GatedAttention`).  Feed-forwards: a sum of normed powers, routed experts beside a gated
shared one, or none (:mod:`~ferrotorch_b200.nn.feed_forward`).  Layers may differ in every size and come in any order.  The model runs
over a paged KV cache with recurrent states only (:class:`~ferrotorch_b200.models.serving.PagedStepper`, ``ContinuousBatcher``,
``generation.generate``)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import torch
from torch import nn

from ..nn.feed_forward import ExpertSpec, PackedMLP, RoutedExperts
from ..nn.gated_attention import GatedAttention, ResidualRMSNorm
from ..nn.packed_block import AttentionSpec, RotarySpec, WavelengthScaling, pad_to, round_up
from ..nn.paged import PagedKVCache, PagedSession, RaggedBatch
from ..nn.recurrent import StateSpaceBlock, StateSpaceSpec, StateSpaceState
from ..ops import decoder as D
from ..ops import functional as F

ARCHITECTURE = "Mogelix"


@dataclass
class MogelixLayerConfig:
    mixer: AttentionSpec | StateSpaceSpec
    mlp: int | ExpertSpec | None = None           # width of a dense feed-forward, experts, or none

    @property
    def is_attention(self) -> bool:
        return isinstance(self.mixer, AttentionSpec)


def _read_rotary(rot: dict | None) -> RotarySpec | None:
    if not rot:
        return None
    s = rot.get("scaling")
    return RotarySpec(int(rot["dims"]), float(rot["base"]),
                      WavelengthScaling(float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"])) if s else None)


def _write_rotary(rot: RotarySpec) -> dict:
    out = {"dims": rot.dims, "base": rot.base}
    if rot.scaling is not None:
        out["scaling"] = dict(vars(rot.scaling))
    return out


@dataclass
class MogelixConfig:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)            # of MogelixLayerConfig
    alpha: float = 1.0                                    # factor of the residual in every sum
    norm_eps: float = 1e-6
    max_position_embeddings: int | None = None            # nothing in the model limits positions

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def experts(experts: int, top: int, ff: int, shared_ff: int | None = None) -> ExpertSpec:
        """Experts by this design's rules: biased logits, softmax over the chosen ones, weights on the outputs, a gated shared expert."""
        return ExpertSpec(experts, top, ff, score="softmax", normalize=True, scale="output", shared_ff=shared_ff, gated=False, router_bias=True,
                          shared_gate=shared_ff is not None)

    @classmethod
    def pattern(cls, vocab_size: int, hidden_size: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, *, window: int = 1024,
                pool: int = 16, state_heads: int | None = None, state_dim: int | None = None, state: int = 128, groups: int = 1, conv: int = 4,
                experts: int = 8, top: int = 2, expert_ff: int | None = None, shared_ff: int | None = None, **kw) -> "MogelixConfig":
        """Layers in groups of six: state space, attention, attention over the keys of the layer before it, state space, attention, state
        space; dense feed-forwards in the first layer of a group and routed ones (``top`` of ``experts``) in the others.  ``experts`` 0:
        all dense."""
        state_dim = state_dim or dim
        state_heads = state_heads or max(1, 2 * hidden_size // state_dim)
        rotary = RotarySpec(dim, 500000.0, WavelengthScaling(8.0, 1.0, 4.0, 8192.0))
        layers = []
        for i in range(n_layers):
            if i % 6 in (1, 2, 4):
                mixer = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window=window, pool=pool, rotary=rotary, kv_from=i - 1 if i % 6 == 2 else None)
            else:
                mixer = StateSpaceSpec(state_heads, state_dim, state, groups, conv, groups)
            routed = experts and i % 6
            layers.append(MogelixLayerConfig(mixer, cls.experts(experts, top, expert_ff or ff // top, shared_ff or ff // top) if routed else ff))
        out = cls(vocab_size, hidden_size, layers, **kw)
        out.validate()
        return out

    @classmethod
    def preset_3b(cls) -> "MogelixConfig":
        """Layer sizes of a model that reads about three billion of its parameters per token (no trained weights exist)."""
        return cls.pattern(128256, 3072, 24, 24, 8, 128, 8192, window=2048, pool=32, state_dim=64, expert_ff=3072, shared_ff=3072, alpha=3.0)

    @classmethod
    def tiny(cls) -> "MogelixConfig":
        """A few layers for smoke tests."""
        return cls.pattern(1000, 128, 6, 4, 2, 32, 192, window=24, pool=8, state_heads=6, state=16, groups=2, experts=4, alpha=2.0)

    @classmethod
    def from_dict(cls, cfg: dict | str) -> "MogelixConfig":
        """Build from a ``config.json`` dict or path."""
        if isinstance(cfg, str):
            with open(cfg) as f:
                cfg = json.load(f)
        if cfg.get("architecture") != ARCHITECTURE:
            raise ValueError("MogelixConfig: architecture is %r" % (cfg.get("architecture"),))
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry.get("type") == "attention":
                mask, source = m.get("mask") or {}, m.get("kv_from")
                mixer = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                      window=int(mask["size"]) if mask.get("size") is not None else None,
                                      pool=int(mask["pool"]) if mask.get("pool") is not None else None, rotary=_read_rotary(m.get("rot")),
                                      kv_from=int(source) if source is not None else None)
            elif entry.get("type") == "mamba2":
                mixer = StateSpaceSpec(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m["norm_groups"]))
            else:
                raise ValueError("MogelixConfig: layer %d has unknown mixer type %r" % (i, entry.get("type")))
            if mlp is None:
                ff = None
            elif mlp.get("kind") == "dense":
                ff = int(mlp["ff"])
            elif mlp.get("kind") == "moe":
                shared = mlp.get("shared")
                ff = cls.experts(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), int(shared["ff"]) if shared else None)
            else:
                raise ValueError("MogelixConfig: layer %d has unknown feed-forward kind %r" % (i, mlp.get("kind")))
            layers.append(MogelixLayerConfig(mixer, ff))
        out = cls(int(cfg["vocab"]), int(cfg["width"]), layers, float(cfg["postln_alpha"]), float(cfg["norm"]["eps"]))
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
                    if a.pool is not None:
                        mixer["mask"]["pool"] = a.pool
                if a.rotary is not None:
                    mixer["rot"] = _write_rotary(a.rotary)
                if a.kv_from is not None:
                    mixer["kv_from"] = a.kv_from
            else:
                mixer = {"heads": a.heads, "vdim": a.vdim, "state": a.state, "groups": a.groups, "conv": a.conv, "norm_groups": a.norm_groups}
            mlp = s.mlp
            if isinstance(mlp, ExpertSpec):
                out = {"kind": "moe", "router": {"experts": mlp.experts, "top": mlp.top}, "expert": {"ff": mlp.ff}}
                if mlp.shared_ff is not None:
                    out["shared"] = {"ff": mlp.shared_ff}
                mlp = out
            elif mlp is not None:
                mlp = {"kind": "dense", "ff": mlp}
            layers.append({"type": "attention" if s.is_attention else "mamba2", "mixer": mixer, "mlp": mlp})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "postln_alpha": self.alpha, "norm": {"eps": self.norm_eps},
                "layers": layers}

    def validate(self) -> None:
        if min(self.vocab_size, self.hidden_size, len(self.layers)) < 1:
            raise ValueError("MogelixConfig: vocabulary, width and layers must be positive")
        for i, s in enumerate(self.layers):
            s.mixer.validate()
            if isinstance(s.mlp, ExpertSpec):
                s.mlp.validate()
            elif s.mlp is not None and s.mlp < 1:
                raise ValueError("MogelixConfig: layer %d: ff must be positive or absent" % i)
            j = s.mixer.kv_from if s.is_attention else None
            if j is not None:
                if not 0 <= j < i or not self.layers[j].is_attention or self.layers[j].mixer.kv_from is not None:
                    raise ValueError("MogelixConfig: layer %d reads the keys of layer %d, which has none ahead of it" % (i, j))
                a, b = s.mixer, self.layers[j].mixer
                if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                    raise ValueError("MogelixConfig: layers %d and %d share keys of different sizes" % (j, i))

    def num_parameters(self) -> int:
        W = self.hidden_size
        total = 2 * self.vocab_size * W + W
        for s in self.layers:
            m = s.mixer
            total += (W * (W + 2)) * (1 if s.mlp is None else 2)
            if s.is_attention:
                total += W * m.heads * (m.dim + m.vdim) + m.heads * (m.dim + 1)
                if m.kv_from is None:
                    total += (W + 1) * m.kv_heads * (m.dim + m.vdim)
            else:
                conv = m.inner + 2 * m.groups * m.state
                total += W * (2 * m.inner + conv + m.heads) + conv * (m.conv + 1) + 3 * m.heads + m.inner
            if isinstance(s.mlp, ExpertSpec):
                e = s.mlp
                total += e.experts * (W + 1 + 2 * W * e.ff) + (W * (2 * e.shared_ff + 1) if e.shared_ff else 0)
            elif s.mlp is not None:
                total += 2 * W * s.mlp + 4
        return total


class MogelixLayer(nn.Module):
    def __init__(self, cfg: MogelixConfig, spec: MogelixLayerConfig):
        super().__init__()
        W, eps = cfg.hidden_size, cfg.norm_eps
        self.norm1 = ResidualRMSNorm(W, eps)
        if spec.is_attention:
            self.mixer = GatedAttention(W, spec.mixer, eps, gate=False, norm_weights=False, bias=True, residual_gate=True)
        else:
            self.mixer = StateSpaceBlock(W, spec.mixer, eps, residual_gate=True)
        self.norm2 = self.mlp = None
        if isinstance(spec.mlp, ExpertSpec):
            self.mlp = RoutedExperts(W, spec.mlp, "relu2", residual_gate=True)
        elif spec.mlp is not None:
            self.mlp = PackedMLP(W, spec.mlp, "poly_norm", eps, residual_gate=True)
        if self.mlp is not None:
            self.norm2 = ResidualRMSNorm(W, eps)

    def parts(self) -> list:
        """``(prefix of the checkpoint names, name of the residual gate, module)`` of the sublayers."""
        return [("mix.", "rg1", self.mixer)] + ([("mlp.", "rg2", self.mlp)] if self.mlp is not None else [])

    def norms(self) -> list:
        return [("norm1", self.norm1)] + ([("norm2", self.norm2)] if self.norm2 is not None else [])


def _checkpoint_name(prefix: str, gate: str, name: str) -> str:
    """The residual gates of a layer stand beside its sublayers."""
    return name.replace("rg", gate, 1) if name in ("rg", "rg.b") else prefix + name


class MogelixForCausalLM(nn.Module):
    """Weights are buffers (inference only).  ``dtype`` of the matrices: bf16 (served) or fp32 (everything in 32-bit); norms,
    the residual, step sizes, decays and states, scores and routing are fp32 in both."""

    def __init__(self, cfg: MogelixConfig, dtype: torch.dtype = torch.bfloat16, device="cpu"):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("MogelixForCausalLM: dtype must be bfloat16 or float32")
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
                layer = MogelixLayer(cfg, s)
                for *_, part in layer.parts():
                    part.cast_(dtype)
                self.layers.append(layer)
            self.final_norm = ResidualRMSNorm(cfg.hidden_size, cfg.norm_eps)
            self.register_buffer("embed", torch.zeros(cfg.vocab_size, width, dtype=dtype))
            self.register_buffer("head", torch.zeros(round_up(cfg.vocab_size, 8), width, dtype=dtype))

    # ------------------------------------------------------------------ weights
    def load_tensors(self, sd: dict) -> None:
        """Load the checkpoint's tensors (names ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.rg1``, ``l<i>.mlp.*``, .., ``final.norm``,
        ``head``); every tensor must be used and have its shape."""
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
            for prefix, gate, module in layer.parts():
                module.load({n: take(pre + _checkpoint_name(prefix, gate, n)) for n in module.tensor_names()})
        if left:
            raise KeyError("checkpoint has tensors this model does not know: %s" % sorted(left)[:8])

    def random_(self, std: float = 0.02, seed: int = 0) -> "MogelixForCausalLM":
        g = torch.Generator(device=self.embed.device).manual_seed(seed)
        c = self.config
        for buf in (self.embed, self.head):
            buf[:c.vocab_size, :c.hidden_size].copy_(torch.randn(c.vocab_size, c.hidden_size, device=buf.device, generator=g) * std)
        for layer in self.layers:
            for *_, part in layer.parts():
                part.random_(std, g)
        return self

    @classmethod
    def tiny_random(cls, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "MogelixForCausalLM":
        return cls(MogelixConfig.tiny(), dtype, device).random_()

    def checkpoint_tensors(self) -> dict:
        """The weights under their checkpoint names, in their true sizes."""
        c = self.config
        out = {"embed": self.embed[:, :c.hidden_size], "head": self.head[:c.vocab_size, :c.hidden_size], "final.norm": self.final_norm.unpack()}
        for i, layer in enumerate(self.layers):
            pre = "l%d." % i
            out.update({pre + name: norm.unpack() for name, norm in layer.norms()})
            for prefix, gate, module in layer.parts():
                out.update({pre + _checkpoint_name(prefix, gate, n): t for n, t in module.unpack().items()})
        return {k: v.contiguous() for k, v in out.items()}

    def save_pretrained(self, path: str) -> None:
        """Write ``config.json`` and ``model.safetensors``."""
        from ..serialize.state import save_safetensors

        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.config.to_dict(), f, indent=1)
        save_safetensors(self.checkpoint_tensors(), os.path.join(path, "model.safetensors"))

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device="cpu") -> "MogelixForCausalLM":
        """The model of a directory with ``config.json`` and ``model.safetensors`` (or shards with an index)."""
        from ..serialize.state import load_safetensors_auto

        model = cls(MogelixConfig.from_dict(os.path.join(path, "config.json")), dtype, device)
        model.load_tensors(load_safetensors_auto(path))
        return model

    # ------------------------------------------------------------------ inference over a paged cache
    def make_paged_cache(self, num_blocks: int, block_size: int, max_seqs: int, max_seq_len: int) -> PagedKVCache:
        """Pages for the layers with keys of their own (and the pooled blocks that any reader of these needs), a state per slot (and one
        for padding rows) for state-space layers."""
        layers = self.config.layers
        specs = [s.mixer for s in layers if s.is_attention and s.mixer.kv_from is None]
        cache = PagedKVCache(len(specs), [a.kv_heads for a in specs], [a.padded_dim for a in specs], num_blocks, max_seqs, max_seq_len,
                             block_size, self.embed.device, self.dtype, v_head_dim=[a.padded_vdim for a in specs])
        for i, place in self._places.items():
            if layers[i].mixer.pool is not None:
                cache.keep_pooled(place, layers[i].mixer.pool)
        cache.states = {i: StateSpaceState(max_seqs + 1, s.mixer, self.embed.device, self.dtype) for i, s in enumerate(layers) if not s.is_attention}
        return cache

    @torch.no_grad()
    def paged_forward(self, batch: RaggedBatch, cache: PagedKVCache, on_layer=None) -> torch.Tensor:
        """One pass over a ragged batch: fp32 logits ``[wanted rows, vocab]``.  ``on_layer(i, x)`` sees the residual (padded width)
        after every layer."""
        c, x, ids = self.config, self.embed, batch.tokens
        h = F.embedding(ids, self.embed)
        end = len(self.layers) - 1
        for i, layer in enumerate(self.layers):
            for module, norm in ((layer.mixer, layer.norm1), (layer.mlp, layer.norm2)):
                if module is None:
                    continue
                if module is layer.mlp:
                    y, gate = module.terms(h)
                elif i in self._places:
                    y, gate = module.terms(h, batch, cache, self._places[i])
                else:
                    y, gate = module.terms(h, batch, cache.states[i])
                kw = dict(count=c.hidden_size, out_dtype=self.dtype, ids=ids)
                if i == end and (module is layer.mlp or layer.mlp is None) and on_layer is None:
                    if batch.n_want:                      # of the last sum only the wanted rows, straight into the final norm
                        _, h = D.sum_norm(x, y, gate, c.alpha, norm.weight, c.norm_eps, rows=batch.last, last=self.final_norm.weight, **kw)
                    continue
                x, h = D.sum_norm(x, y, gate, c.alpha, norm.weight, c.norm_eps, **kw)
                ids = None
            if on_layer is not None:
                on_layer(i, x)
        if batch.n_want == 0:
            return torch.empty((0, c.vocab_size), device=x.device)
        if on_layer is not None:
            h = self.final_norm(x, rows=batch.last, out_dtype=self.dtype)
        return F.linear_f32_out(h, self.head)[:, :c.vocab_size]

    # ------------------------------------------------------------------ dense entry points (models.generation)
    def make_caches(self, batch: int, max_len: int, device=None, dtype=None) -> PagedSession:
        return PagedSession(self, batch, max_len)

    def forward(self, input_ids: torch.Tensor, *, caches: PagedSession | None = None, last_token_only: bool = False) -> torch.Tensor:
        """Logits ``[B, S, vocab]`` (or ``[B, 1, vocab]``) of equally long sequences, continuing ``caches`` when given."""
        session = caches if caches is not None else PagedSession(self, *input_ids.shape)
        return session.extend(input_ids, last_token_only)

"""Small Zolorax configurations with random weights.

Weights are bf16 values (so both number formats start from the same numbers).  Score scales and sinks make attention peaky,
decays range from a few to hundreds of tokens, and router logits are spread out, so that a wrong, missing or foreign key,
state or expert shows in the logits."""
import copy

import torch

import zolorax_oracle as O
from decoder_cases import VOCAB, DecoderCase
from ferrotorch_b200.models.zolorax import ZoloraxConfig, ZoloraxForCausalLM


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def attention(heads, kv, dim, vdim, window, mlp, rot=8, base=300.0, factor=3.0, original=60, fast=4.0, slow=0.5, sharp=2.5, source=None):
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": sharp / dim ** 0.5,
             "rot": {"base": base, "dims": rot, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}
    if source is not None:
        mixer["kv_from"] = source
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def recurrent(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


# sizes that are equal or 1 in ordinary models differ here: key and value heads, groups, windows of sharing layers,
# recurrent widths, blocks that are no multiple of 8, one tap or many, layers without a feed-forward, any order
CASES = {
    "mixed": dict(width=52, eps=1e-5, layers=[
        recurrent(36, 3, 4, dense(60)), attention(6, 2, 24, 40, 9, moe(5, 2, 20), rot=16),
        attention(4, 2, 24, 40, 21, None, rot=16, source=1), recurrent(80, 1, 1, moe(8, 1, 33)), attention(3, 3, 12, 8, 64, dense(17), rot=4)]),
    "recurrent": dict(width=40, eps=1e-3, layers=[recurrent(48, 2, 2, moe(3, 3, 16)), recurrent(24, 4, 6, None), recurrent(128, 2, 3, dense(41))]),
    "attention": dict(width=64, eps=1e-6, layers=[
        attention(4, 4, 32, 32, 16, dense(96), rot=32, factor=1.0), attention(4, 1, 64, 64, 1, moe(40, 4, 8), rot=64, base=1000.0),
        attention(8, 1, 64, 64, 33, moe(2, 1, 24), rot=64, base=1000.0, source=1), attention(2, 1, 64, 64, 130, dense(32), rot=64, source=1)]),
    "wide heads": dict(width=24, eps=1e-4, layers=[attention(2, 1, 72, 100, 40, dense(40), rot=2, original=1000), recurrent(40, 5, 3, dense(8)),
                                                   attention(1, 1, 144, 16, 30, moe(6, 2, 12), rot=144, fast=32.0, slow=1.0)]),
}


def config_dict(case) -> dict:
    c = copy.deepcopy(CASES[case])
    return {"architecture": "Zolorax", "vocab": VOCAB, "width": c["width"], "norm": {"eps": c["eps"]}, "layers": c["layers"]}


def random_weights(cfg: dict, seed: int = 0, spread: float = 1.0) -> dict:
    """``spread``: how much the experts of a layer differ.  In bf16 two experts with nearly equal scores may change places
    with the rounding of their input, so tests of whole models in bf16 use experts that are alike."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).bfloat16()

    out = {"embed": rnd(V, W), "head": rnd(V, W, std=W ** -0.5), "final.norm": rnd(W, std=0.2)}
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, pre = entry["mixer"], entry["mlp"], "l%d." % i
        mix, ff = pre + "mix.", pre + "mlp."
        out[pre + "norm1"] = rnd(W, std=0.3)
        if entry["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[mix + "q"], out[mix + "g"] = rnd(H * D, W, std=W ** -0.5), rnd(H * Dv, W, std=W ** -0.5)
            out[mix + "q.norm"], out[mix + "sink"] = rnd(D, std=0.2, mean=1.0), rnd(H, std=1.5, mean=1.0)
            out[mix + "o"] = rnd(W, H * Dv, std=2.0 * (H * Dv) ** -0.5)
            if "kv_from" not in m:
                out[mix + "k"], out[mix + "v"] = rnd(G * D, W, std=W ** -0.5), rnd(G * Dv, W, std=W ** -0.5)
                out[mix + "k.norm"] = rnd(D, std=0.2, mean=1.0)
        else:
            w, n = m["width"], m["width"] // m["blocks"]
            for name in ("y", "x"):
                out[mix + name], out[mix + name + ".b"] = rnd(w, W, std=W ** -0.5), rnd(w, std=0.3)
            out[mix + "conv"], out[mix + "conv.b"] = rnd(w, m["conv"], std=0.6), rnd(w, std=0.2)
            for name in ("ra", "ri"):
                out[mix + name], out[mix + name + ".b"] = rnd(m["blocks"], n, n, std=n ** -0.5), rnd(m["blocks"], n, std=0.5)
            out[mix + "lam"] = (torch.rand(w, generator=g) * 7.0 - 6.0).bfloat16()
            out[mix + "o"] = rnd(W, w, std=1.5 * w ** -0.5)
        if mlp is None:
            continue
        out[pre + "norm2"] = rnd(W, std=0.3)
        if mlp["kind"] == "dense":
            out[ff + "up"], out[ff + "down"] = rnd(mlp["ff"], W, std=W ** -0.5), rnd(W, mlp["ff"], std=mlp["ff"] ** -0.5)
            continue
        n, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        out[ff + "router"] = rnd(E, W, std=2.0 * W ** -0.5)
        for name, shape in (("gate", (n, W)), ("up", (n, W)), ("down", (W, n))):
            common = torch.randn(shape, generator=g)
            for e in range(E):
                own = torch.randn(shape, generator=g)
                mixed = spread * own + (1.0 - spread) * common
                out[ff + "e%d.%s" % (e, name)] = (mixed / (spread ** 2 + (1 - spread) ** 2) ** 0.5 * 1.5 * shape[1] ** -0.5).bfloat16()
    return out


class Case(DecoderCase):
    def __init__(self, name: str, dtype=torch.float32, device="cpu", seed: int = 1):
        cfg = config_dict(name)
        weights = random_weights(cfg, seed, 1.0 if dtype == torch.float32 else 0.05)
        if dtype != torch.float32:                        # rounded queries and keys: scores of tens would carry errors of tenths
            for entry in cfg["layers"]:
                if entry["type"] == "attention":
                    entry["mixer"]["scale"] *= 0.4
        super().__init__(cfg, weights, ZoloraxForCausalLM(ZoloraxConfig.from_dict(cfg), dtype, device), O.forward)
        self.loose_rows = 0.0 if dtype == torch.float32 else 0.05      # an expert may still change places

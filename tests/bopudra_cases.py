"""Small Bopudra configurations with random weights.

Weights are bf16 values (so both number formats start from the same numbers) with norms, temperatures and score scales
that make attention peaky: a single key carries much of a softmax, so a wrong, missing or foreign key shows in the
logits."""
import copy

import torch

import bopudra_oracle as O
from decoder_cases import (VOCAB, DecoderCase, check_batches, check_generation, check_portions, check_whole_prompt, feed_all,  # noqa: F401
                           greedy)
from ferrotorch_b200.models.bopudra import BopudraConfig, BopudraForCausalLM


def layer(heads, kv, dim, vdim, ff, coef=0.4, every=7, sharp=2.5):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": sharp / dim ** 0.5,
                                           "q_temp": {"coef": coef, "every": every}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


# sizes that are equal or 1 in ordinary models differ here: key and value heads, layers, groups of 1 / 3 / 5 / 6, odd widths
CASES = {
    "even": dict(width=64, logit_scale=0.75, eps=1e-5, layers=[layer(4, 2, 32, 32, 96), layer(4, 2, 32, 32, 96)]),
    "uneven": dict(width=52, logit_scale=3.0, eps=1e-3, layers=[layer(6, 2, 24, 40, 60, 0.9, 5), layer(5, 1, 12, 20, None, 0.3, 16),
                                                                layer(3, 3, 36, 8, 33, 0.0, 1), layer(6, 1, 72, 100, 50, 0.25, 64)]),
    "one head": dict(width=24, logit_scale=1.0, eps=1e-6, layers=[layer(1, 1, 16, 64, 40, 1.5, 2), layer(2, 1, 80, 16, 17, 0.1, 3)]),
}


def config_dict(case) -> dict:
    c = copy.deepcopy(CASES[case])
    return {"architecture": "Bopudra", "vocab": VOCAB, "width": c["width"], "logit_scale": c["logit_scale"], "norm": {"eps": c["eps"]},
            "layers": c["layers"]}


def random_weights(cfg: dict, seed: int = 0) -> dict:
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).bfloat16()

    def norm(out, name):
        out[name], out[name + ".b"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.2)
        out[name + ".alpha"] = (torch.rand((), generator=g) * 0.8 + 0.4).bfloat16()

    out = {"embed": rnd(V, W), "head": rnd(V, W, std=W ** -0.5)}
    norm(out, "final.norm")
    for i, entry in enumerate(cfg["layers"]):
        m, pre = entry["mixer"], "l%d." % i
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(out, pre + "norm1")
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv), ("g", H)):
            out[pre + "mix." + n] = rnd(rows, W, std=W ** -0.5)
        out[pre + "mix.o"] = rnd(W, H * Dv, std=1.5 * (H * Dv) ** -0.5)
        out[pre + "mix.q.norm"], out[pre + "mix.k.norm"] = rnd(H * D, std=0.2, mean=1.0), rnd(G * D, std=0.2, mean=1.0)
        if entry["mlp"]:
            ff = entry["mlp"]["ff"]
            out[pre + "mlp.up"], out[pre + "mlp.down"] = rnd(ff, W, std=W ** -0.5), rnd(W, ff, std=ff ** -0.5)
    return out


class Case(DecoderCase):
    def __init__(self, name: str, dtype=torch.float32, device="cpu", seed: int = 0):
        cfg = config_dict(name)
        super().__init__(cfg, random_weights(cfg, seed), BopudraForCausalLM(BopudraConfig.from_dict(cfg), dtype, device), O.forward)

"""Small Mogelix configurations with random weights.

Weights are bf16 values (so both number formats start from the same numbers).  Scores are peaky, decays keep states for a few to
hundreds of tokens, and router logits are spread out, so that a wrong, missing or foreign key, block, state or expert shows in the
logits."""
import copy

import torch

import mogelix_oracle as O
from decoder_cases import VOCAB, DecoderCase
from ferrotorch_b200.models.mogelix import MogelixConfig, MogelixForCausalLM


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}


def ssd(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def att(heads, kv, dim, vdim, mask, rot, mlp, kv_from=None, sharp=6.0):
    """Queries and keys have unit mean square, so scores are about ``sharp`` at most; ``rot``: (dims, base, scaling or None)."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": sharp / dim}
    if mask:
        m["mask"] = dict(zip(("size", "pool"), mask))
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1], **({"scaling": dict(zip(("factor", "low", "high", "original"), rot[2]))} if rot[2] else {})}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


SCALED = (3.0, 1.5, 5.0, 40)     # some frequencies of a rotation with a small base lie on either side and between

# sizes that are equal or 1 in ordinary models differ here: key and value heads, groups of heads, of states and of norms (whose parts
# cut through heads), taps, windows, blocks smaller and larger than a page, readers with blocks of their own, any order
CASES = {
    "mixed": dict(width=52, eps=1e-5, alpha=1.7, layers=[
        att(6, 2, 24, 40, (9, 4), (16, 30.0, SCALED), dense(67)), ssd(6, 20, 12, 2, 3, 4, moe(5, 2, 20, 33)),
        att(2, 2, 24, 40, (14, 5), (24, 100.0, None), None, kv_from=0), att(3, 3, 12, 8, (5, 20), None, moe(4, 4, 17)),
        ssd(1, 33, 40, 1, 1, 3, None), att(4, 2, 24, 40, (7, 1), (8, 30.0, SCALED), moe(6, 1, 9, 8), kv_from=0)]),
    "state": dict(width=40, eps=1e-3, alpha=1.4, layers=[
        ssd(4, 16, 32, 1, 4, 1, dense(24)), ssd(3, 8, 7, 3, 5, 1, moe(3, 2, 16, 24)), ssd(8, 32, 16, 4, 2, 8, dense(200))]),
    "attention": dict(width=64, eps=1e-6, alpha=2.5, layers=[
        att(4, 4, 32, 32, (16, 16), (32, 50.0, SCALED), dense(48)), att(8, 2, 64, 64, (1, 3), None, moe(40, 4, 8, 16)),
        att(8, 1, 16, 48, (30, 2), (16, 500.0, None), dense(96)), att(2, 1, 16, 48, None, (16, 500.0, None), None, kv_from=2),
        att(4, 2, 32, 16, (12,), (32, 30.0, SCALED), moe(7, 3, 24))]),
    "wide heads": dict(width=24, eps=1e-4, alpha=0.8, layers=[
        att(2, 1, 144, 100, (20, 6), (100, 80.0, SCALED), dense(8)), ssd(2, 272, 136, 1, 4, 2, moe(2, 1, 12, 8)),
        att(18, 1, 32, 24, (11, 7), (32, 60.0, None), None), ssd(2, 24, 8, 2, 7, 1, dense(33))]),
}


def config_dict(case) -> dict:
    c = copy.deepcopy(CASES[case])
    return {"architecture": "Mogelix", "vocab": VOCAB, "width": c["width"], "norm": {"eps": c["eps"]}, "postln_alpha": c["alpha"], "layers": c["layers"]}


def random_weights(cfg: dict, seed: int = 0, close_calls: bool = True) -> dict:
    """Without ``close_calls`` the biases of the router are far apart, so that the rounding of its input in bf16 changes no choice, and
    no head's skip is small: where a head's states nearly cancel against C, a norm over that head alone would magnify their
    rounding.  Tests of whole models in bf16 use that."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).bfloat16()

    out = {"embed": rnd(V, W), "head": rnd(V, W, std=2.0 * W ** -0.5), "final.norm": rnd(W, std=0.2, mean=1.0)}
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, pre = entry["mixer"], entry["mlp"], "l%d." % i
        mix, ff = pre + "mix.", pre + "mlp."
        for n in ("1", "2") if mlp else ("1",):
            out[pre + "norm" + n] = rnd(W, std=0.3, mean=1.0)
            out[pre + "rg" + n], out[pre + "rg%s.b" % n] = rnd(W, W, std=W ** -0.5), rnd(W, std=0.5, mean=1.0)
        if entry["type"] == "mamba2":
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner, conv = H * P, H * P + 2 * G * N
            out[mix + "in"] = rnd(inner + conv + H, W, std=W ** -0.5)
            out[mix + "conv"], out[mix + "conv.b"] = rnd(conv, m["conv"], std=m["conv"] ** -0.5), rnd(conv, std=0.3)
            out[mix + "dt_bias"], out[mix + "A_log"], out[mix + "D"] = rnd(H, mean=-2.0), rnd(H, std=1.5, mean=-1.0), rnd(H, std=0.5 if close_calls else 0.2, mean=0.5 if close_calls else 2.0)
            out[mix + "norm"], out[mix + "o"] = rnd(inner, std=0.3, mean=1.0), rnd(W, inner, std=2.0 * inner ** -0.5)
        else:
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, n in (("q", H * D),) + ((("k", G * D), ("v", G * Dv)) if "kv_from" not in m else ()):
                out[mix + name], out[mix + name + ".b"] = rnd(n, W, std=W ** -0.5), rnd(n, std=0.5)
            out[mix + "o"], out[mix + "sink"] = rnd(W, H * Dv, std=2.0 * (H * Dv) ** -0.5), rnd(H)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out[ff + "up"], out[ff + "down"] = rnd(mlp["ff"], W, std=W ** -0.5), rnd(W, mlp["ff"], std=1.5 * mlp["ff"] ** -0.5)
            out[ff + "act"] = rnd(4, std=0.3) + torch.tensor([0.8, 0.5, -0.4, 0.2]).bfloat16()
            continue
        r = mlp["router"]
        out[ff + "router"] = rnd(r["experts"], W, std=(1.5 if close_calls else 1.0) * W ** -0.5)
        out[ff + "router.b"] = rnd(r["experts"]) if close_calls else (torch.randperm(r["experts"], generator=g) * 8.0).bfloat16()
        shared = mlp.get("shared")
        for name, width in [("e%d" % e, mlp["expert"]["ff"]) for e in range(r["experts"])] + ([("shared", shared["ff"])] if shared else []):
            out[ff + name + ".up"], out[ff + name + ".down"] = rnd(width, W, std=1.5 * W ** -0.5), rnd(W, width, std=width ** -0.5)
        if shared:
            out[ff + "shared.sg"] = rnd(1, W, std=2.0 * W ** -0.5)
    return out


class Case(DecoderCase):
    def __init__(self, name: str, dtype=torch.float32, device="cpu", seed: int = 1):
        cfg = config_dict(name)
        if dtype != torch.float32:                        # rounded queries and keys: scores of many would carry errors of hundredths
            for entry in cfg["layers"]:
                if entry["type"] == "attention":
                    entry["mixer"]["scale"] *= 0.5
        weights = random_weights(cfg, seed, dtype == torch.float32)
        super().__init__(cfg, weights, MogelixForCausalLM(MogelixConfig.from_dict(cfg), dtype, device), O.forward)
        if dtype != torch.float32:                        # norms over parts of a dozen elements, cubes and squares magnify rounding here and there
            self.loose_rows, self.tolerance = 0.05, 0.08

"""Small Tenalorn configurations with random weights.

Weights are bf16 values (so both number formats start from the same numbers).  Score scales make attention peaky, forget
gates keep memories for a few to hundreds of tokens, and router scores are spread out, so that a wrong, missing or foreign
key, state, previous token or expert shows in the logits."""
import copy

import torch

import tenalorn_oracle as O
from decoder_cases import VOCAB, DecoderCase
from ferrotorch_b200.models.tenalorn import TenalornConfig, TenalornForCausalLM


def moe(experts, top, ff, identity=0, shared=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}, "shared": {"ff": shared}}


def parallel(heads, kv, dim, vdim, chunk, memory, mlp, cap=6.0, left=0.8, right=1.3, sharp=6.0):
    """``memory``: heads, dim, vdim.  Queries and keys have unit mean square, so scores are about ``sharp`` at most."""
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": sharp / dim},
        "right": {"heads": memory[0], "dim": memory[1], "vdim": memory[2], "gate_cap": cap}, "left_scale": left, "right_scale": right}}


def latent(heads, dim, rot, vdim, rank, mlp, base=300.0, sharp=2.5, dims=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                            "scale": sharp / (dim + rot) ** 0.5, "rot": {"base": base, "dims": dims or rot}}}


# sizes that are equal or 1 in ordinary models differ here: key and value heads, groups, chunks, memory sizes, rotated and
# unrotated parts, ranks that are no multiple of 16, experts' and shared widths, one stream or many, any order
CASES = {
    "mixed": dict(width=52, eps=1e-5, streams=3, scale=1.5, cap=9.0, bigram=(101, 31, 7), layers=[
        parallel(6, 2, 24, 40, 9, (3, 20, 12), moe(5, 2, 20, 2)), latent(5, 20, 6, 24, 36, moe(8, 3, 33, 1, 40)),
        parallel(3, 3, 12, 8, 21, (1, 40, 64), None, cap=15.0, left=1.0, right=1.0), latent(2, 12, 16, 72, 20, None),
        parallel(4, 1, 64, 64, 64, (2, 33, 24), moe(3, 1, 17, 0, 8), cap=2.0)]),
    "latent": dict(width=40, eps=1e-3, streams=1, scale=0.7, cap=30.0, bigram=(7, 2, 3), layers=[
        latent(4, 32, 32, 32, 64, moe(4, 4, 16, 1)), latent(1, 8, 2, 40, 10, moe(2, 2, 24, 3, 33)), latent(9, 16, 8, 16, 96, None)]),
    "parallel": dict(width=64, eps=1e-6, streams=5, scale=1.0, cap=15.0, bigram=(1021, 5, 1), layers=[
        parallel(4, 4, 32, 32, 16, (4, 32, 32), moe(6, 2, 48, 2)), parallel(4, 2, 64, 64, 1, (2, 64, 128), None),
        parallel(8, 2, 16, 48, 130, (1, 16, 16), moe(40, 4, 8, 8, 16), left=0.3, right=2.0)]),
    "wide heads": dict(width=24, eps=1e-4, streams=2, scale=3.0, cap=5.0, bigram=(64, 9, 4), layers=[
        parallel(2, 1, 144, 100, 40, (1, 136, 272), moe(3, 2, 12, 1)), latent(18, 100, 60, 130, 200, moe(2, 1, 8, 1, 12)),
        parallel(1, 1, 8, 160, 33, (2, 24, 8), None)]),
}


def config_dict(case) -> dict:
    c = copy.deepcopy(CASES[case])
    big = dict(zip(("buckets", "mul_prev", "mul_cur"), c["bigram"]))
    return {"architecture": "Tenalorn", "vocab": VOCAB, "width": c["width"], "streams": c["streams"], "norm": {"eps": c["eps"]}, "logit_softcap": c["cap"],
            "embedding": {"scale": c["scale"], "bigram": big}, "layers": c["layers"]}


def random_weights(cfg: dict, seed: int = 0, close_calls: bool = True) -> dict:
    """Without ``close_calls`` the corrections of the router are far apart, so that the rounding of its input in bf16 changes
    no choice, and the keys of memories resemble their queries: the direction of a memory's output hangs on the sign of
    n.q, which rounding may turn where it is nearly zero.  Tests of whole models in bf16 use that."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).bfloat16()

    out = {"embed": rnd(V, W), "bigram": rnd(cfg["embedding"]["bigram"]["buckets"] + 1, W), "head": rnd(V, W, std=2.0 * W ** -0.5), "final.norm": rnd(W, std=0.2, mean=1.0)}
    for i, entry in enumerate(cfg["layers"]):
        m, mlp, pre = entry["mixer"], entry["mlp"], "l%d." % i
        mix, ff = pre + "mix.", pre + "mlp."
        for q in ("1", "2") if mlp else ("1",):
            out[pre + "norm" + q] = rnd(W, std=0.3, mean=1.0)
            out[pre + "hc%s.in" % q], out[pre + "hc%s.out" % q] = rnd(S, std=0.3, mean=0.7), rnd(S, std=0.4, mean=0.8)
            out[pre + "hc%s.mix" % q] = (0.8 * torch.eye(S) + 0.25 * torch.randn(S, S, generator=g)).bfloat16()
        if entry["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for name, shape in (("q", (H * D, W)), ("k", (G * D, W)), ("v", (G * Dv, W))):
                out[mix + "left." + name] = rnd(*shape, std=W ** -0.5)
            out[mix + "left.o"] = rnd(W, H * Dv, std=2.0 * (H * Dv) ** -0.5)
            H, D, Dv = b["heads"], b["dim"], b["vdim"]
            for name, shape in (("q", (H * D, W)), ("k", (H * D, W)), ("v", (H * Dv, W)), ("g", (H * Dv, W)), ("i", (H, W)), ("f", (H, W))):
                out[mix + "right." + name] = rnd(*shape, std=W ** -0.5)
            if not close_calls:
                out[mix + "right.k"] = (0.95 * out[mix + "right.q"].float() + 0.3 * out[mix + "right.k"].float()).bfloat16()
            out[mix + "right.o"], out[mix + "right.norm"] = rnd(W, H * Dv, std=2.0 * (H * Dv) ** -0.5), rnd(H * Dv, std=0.3, mean=1.0)
            out[mix + "right.i.b"], out[mix + "right.f.b"] = rnd(H), rnd(H, std=1.5, mean=3.0)
        else:
            H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            for name, shape in (("q", (H * (D + R), W)), ("dkv", (rank + R, W)), ("g", (H * Dv, W))):
                out[mix + name] = rnd(*shape, std=W ** -0.5)
            out[mix + "dkv.norm"] = rnd(rank, std=0.2, mean=1.0)
            out[mix + "uk"], out[mix + "uv"] = rnd(H * D, rank, std=rank ** -0.5), rnd(H * Dv, rank, std=rank ** -0.5)
            out[mix + "o"] = rnd(W, H * Dv, std=3.0 * (H * Dv) ** -0.5)
        if mlp is None:
            continue
        r = mlp["router"]
        n = r["experts"] + r["identity"]
        out[ff + "router"] = rnd(n, W, std=(1.5 if close_calls else 1.0) * W ** -0.5)
        out[ff + "correction"] = rnd(n, std=0.1) if close_calls else (torch.randperm(n, generator=g) * 2.0).bfloat16()
        for name, width in [("e%d" % e, mlp["expert"]["ff"]) for e in range(r["experts"])] + [("shared", mlp["shared"]["ff"])]:
            out[ff + name + ".gate"], out[ff + name + ".up"] = rnd(width, W, std=1.5 * W ** -0.5), rnd(width, W, std=1.5 * W ** -0.5)
            out[ff + name + ".down"] = rnd(W, width, std=1.5 * width ** -0.5)
    return out


class Case(DecoderCase):
    def __init__(self, name: str, dtype=torch.float32, device="cpu", seed: int = 1):
        cfg = config_dict(name)
        if dtype != torch.float32:                        # rounded queries and keys: scores of tens would carry errors of tenths
            for entry in cfg["layers"]:
                m = entry["mixer"].get("left", entry["mixer"])
                m["scale"] *= 0.5
        weights = random_weights(cfg, seed, dtype == torch.float32)
        super().__init__(cfg, weights, TenalornForCausalLM(TenalornConfig.from_dict(cfg), dtype, device), O.forward)
        self.loose_rows = 0.0 if dtype == torch.float32 else 0.05

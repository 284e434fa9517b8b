"""Plain, slow restatement of the Mogelix decoder: one function per mechanism, written from its equations in 64-bit torch
on the CPU, one sequence at a time.  Shares no code with the package; the tests compare against it.

Notation: a sequence has tokens t = 0 .. T-1; W.. are ``[out, in]`` matrices, b.. biases; the residual is ``[T, width]``."""
import math

import torch


def rms(z, eps):
    """z / sqrt(mean(z^2) + eps) along the last axis."""
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------ residual
def gated(y, h, W, b):
    """A sublayer's output times its gate, which is computed from the sublayer's input."""
    return y * torch.sigmoid(h @ W.T + b)


def normed_sum(x, y, alpha, weight, eps):
    return rms(alpha * x + y, eps) * weight


# ------------------------------------------------------------------ state-space mixer
def causal_conv(z, weight, bias):
    """``z [T, C]``, ``weight [C, taps]`` (its last column meets the token itself), zeros ahead of the sequence."""
    T, taps = z.shape[0], weight.shape[1]
    out = torch.zeros_like(z)
    for t in range(T):
        out[t] = bias
        for d in range(taps):
            if t - d >= 0:
                out[t] = out[t] + weight[:, taps - 1 - d] * z[t - d]
    return out


def state_space(x, B, C, step, rate, skip):
    """One head: ``x [T, vdim]``, ``B, C [T, N]``, step sizes ``step [T]`` > 0, decay rate ``rate`` > 0 -> ``[T, vdim]``.

    S <- e^(-rate step) S + step B x^T from S = 0; output S^T C + skip x."""
    S, out = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype), []
    for t in range(x.shape[0]):
        S = torch.exp(-rate * step[t]) * S + step[t] * torch.outer(B[t], x[t])
        out.append(S.T @ C[t] + skip * x[t])
    return torch.stack(out)


def parts_rms(z, parts, eps):
    """Each of ``parts`` equal runs of the last axis over its own root mean square."""
    return rms(z.unflatten(-1, (parts, -1)), eps).flatten(-2)


def ssd_mixer(h, W, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = (h @ W["in"].T).split([inner, inner + 2 * G * N, H], 1)
    x, B, C = silu(causal_conv(xbc, W["conv"], W["conv.b"])).split([inner, G * N, G * N], 1)
    step, rate = softplus(dt + W["dt_bias"]), torch.exp(W["A_log"])
    y = []
    for a in range(H):
        g = a // (H // G)
        y.append(state_space(x[:, a * P:(a + 1) * P], B[:, g * N:(g + 1) * N], C[:, g * N:(g + 1) * N], step[:, a], rate[a], W["D"][a]))
    return (parts_rms(torch.cat(y, 1) * silu(z), m["norm_groups"], eps) * W["norm"]) @ W["o"].T


# ------------------------------------------------------------------ attention over a window and pooled blocks
def frequencies(rot):
    """base^(-2i / dims), slow ones divided by a factor with a linear transition (in turns over the original length)."""
    out, sc = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_halves(z, position, rot):
    """Elements i and i + dims / 2 turn by position * f_i; those behind the first ``dims`` stay."""
    half = rot["dims"] // 2
    a = (position * frequencies(rot)).to(z.dtype)
    u, v = z[:half], z[half:2 * half]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), z[2 * half:]])


def visible_blocks(position, size, pool):
    """How many pooled blocks a query sees: those that end at or ahead of ``position - size``."""
    n = 0
    while n * pool + pool - 1 <= position - size:
        n += 1
    return n


def windowed_attention(q, keys, values, scale, sink, position, size=None, pool=None):
    """One query over the last ``size`` positions and the means of the blocks ahead of them, one softmax with a sink."""
    first = 0 if size is None else max(0, position - size + 1)
    k, v = list(keys[first:position + 1]), list(values[first:position + 1])
    for b in range(visible_blocks(position, size, pool) if pool else 0):
        k.append(keys[b * pool:(b + 1) * pool].mean(0))
        v.append(values[b * pool:(b + 1) * pool].mean(0))
    s = torch.stack(k) @ q * scale
    top = torch.maximum(s.max(), sink)
    w = torch.exp(s - top)
    return (w / (w.sum() + torch.exp(sink - top))) @ torch.stack(v)


def project_heads(h, W, name, heads, dim):
    return (h @ W[name].T + W[name + ".b"]).view(h.shape[0], heads, dim)


def finish_heads(z, rot, eps):
    """Rotation, then every head over its root mean square."""
    if rot:
        z = torch.stack([torch.stack([rotate_halves(u, t, rot) for u in row]) for t, row in enumerate(z)])
    return rms(z, eps)


def attention_mixer(h, W, m, eps, shared=None):
    """``shared``: keys and values of another layer.  Returns the output and the keys and values that were used."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    mask, rot = m.get("mask") or {}, m.get("rot")
    q = finish_heads(project_heads(h, W, "q", H, m["dim"]), rot, eps)
    k, v = shared if shared is not None else (finish_heads(project_heads(h, W, "k", G, m["dim"]), rot, eps), project_heads(h, W, "v", G, m["vdim"]))
    out = []
    for t in range(T):
        out.append(torch.cat([windowed_attention(q[t, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], W["sink"][a], t, mask.get("size"), mask.get("pool"))
                              for a in range(H)]))
    return torch.stack(out) @ W["o"].T, (k, v)


# ------------------------------------------------------------------ feed-forward
def poly_norm(z, a, b, c, e, eps):
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, W, eps):
    return poly_norm(h @ W["up"].T, *W["act"], eps) @ W["down"].T


def expert(h, W):
    return torch.clamp(h @ W["up"].T, min=0.0) ** 2 @ W["down"].T


def route(logits, top):
    """The ``top`` largest logits and the softmax over these alone."""
    chosen = sorted(range(len(logits)), key=lambda e: -logits[e])[:top]
    w = [math.exp(logits[e] - logits[chosen[0]]) for e in chosen]
    return [(e, u / sum(w)) for e, u in zip(chosen, w)]


def mixture(h, W, mlp):
    z = h @ W["router"].T + W["router.b"]
    out = torch.zeros_like(h)
    if mlp.get("shared"):
        out = expert(h, _sub(W, "shared.")) * torch.sigmoid(h @ W["shared.sg"].T)
    for t in range(h.shape[0]):
        for e, w in route(z[t].tolist(), mlp["router"]["top"]):
            out[t] = out[t] + w * expert(h[t], _sub(W, "e%d." % e))
    return out


# ------------------------------------------------------------------ the model
def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, every_layer=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the residual after every layer)."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x, after, cached = W["embed"][torch.as_tensor(tokens)], [], {}
    for n, layer in enumerate(config["layers"]):
        w, m = _sub(W, "l%d." % n), layer["mixer"]
        if layer["type"] == "attention":
            y, cached[n] = attention_mixer(x, _sub(w, "mix."), m, eps, cached[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = ssd_mixer(x, _sub(w, "mix."), m, eps)
        x = normed_sum(x, gated(y, x, w["rg1"], w["rg1.b"]), alpha, w["norm1"], eps)
        if layer["mlp"] is not None:
            ff = _sub(w, "mlp.")
            y = dense(x, ff, eps) if layer["mlp"]["kind"] == "dense" else mixture(x, ff, layer["mlp"])
            x = normed_sum(x, gated(y, x, w["rg2"], w["rg2.b"]), alpha, w["norm2"], eps)
        after.append(x)
    logits = (rms(x, eps) * W["final.norm"]) @ W["head"].T
    return (logits, after) if every_layer else logits

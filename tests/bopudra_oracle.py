"""Plain, slow restatement of the Bopudra decoder: one function per mechanism, written from its equations in 64-bit
torch on the CPU, one sequence at a time.  Shares no code with the package; the tests compare against it.

Notation: a sequence has tokens t = 0 .. T-1 with residual x_t; W.. are ``[out, in]`` matrices."""
import math

import torch


def dynamic_tanh(x, alpha, weight, bias):
    """tanh(alpha x) * w + b, element by element."""
    return torch.tanh(alpha * x) * weight + bias


def rms_over_all(z, weight, eps):
    """z / sqrt(mean(z^2) + eps) * w over the whole row of a projection, before it is cut into heads."""
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps) * weight


def query_temperature(position, coef, every):
    """1 + coef * ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def head_attention(q, keys, values, scale):
    """One query ``[dim]`` of one head over its visible keys ``[n, dim]`` / values ``[n, vdim]``: softmax of the scaled products."""
    s = keys @ q * scale
    w = torch.exp(s - s.max())
    return (w / w.sum()) @ values


def attention_mixer(h, W, mixer, eps):
    """``h [T, width]`` -> ``[T, width]``.  W: q, k, v, q.norm, k.norm, g, o."""
    T = h.shape[0]
    H, G, D, Dv = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = rms_over_all(h @ W["q"].T, W["q.norm"], eps)
    k = rms_over_all(h @ W["k"].T, W["k.norm"], eps)
    v = h @ W["v"].T
    gate = torch.sigmoid(h @ W["g"].T)
    out = torch.zeros(T, H * Dv, dtype=h.dtype)
    for t in range(T):
        qt = q[t] * query_temperature(t, mixer["q_temp"]["coef"], mixer["q_temp"]["every"])
        for a in range(H):
            c = a // (H // G)
            o = head_attention(qt[a * D:(a + 1) * D], k[:t + 1, c * D:(c + 1) * D], v[:t + 1, c * Dv:(c + 1) * Dv], mixer["scale"])
            out[t, a * Dv:(a + 1) * Dv] = o * gate[t, a]
    return out @ W["o"].T


def feed_forward(h, W):
    return gelu_tanh(h @ W["up"].T) @ W["down"].T


def parallel_layer(x, i, layer, W, eps):
    """x + mixer(h) + ff(h) with one h = norm(x)."""
    pre = "l%d." % i
    h = dynamic_tanh(x, W[pre + "norm1.alpha"], W[pre + "norm1"], W[pre + "norm1.b"])
    y = attention_mixer(h, {n: W[pre + "mix." + n] for n in ("q", "k", "v", "q.norm", "k.norm", "g", "o")}, layer["mixer"], eps)
    if layer["mlp"] is not None:
        y = y + feed_forward(h, {n: W[pre + "mlp." + n] for n in ("up", "down")})
    return x + y


def forward(config, weights, tokens, dtype=torch.float64, every_layer=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the residual after every layer)."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(config["layers"]):
        x = parallel_layer(x, i, layer, W, config["norm"]["eps"])
        after.append(x)
    h = dynamic_tanh(x, W["final.norm.alpha"], W["final.norm"], W["final.norm.b"])
    logits = h @ W["head"].T * config["logit_scale"]
    return (logits, after) if every_layer else logits

"""Plain, slow restatement of the Zolorax decoder: one function per mechanism, written from its equations in 64-bit torch
on the CPU, one sequence at a time.  Shares no code with the package; the tests compare against it.

Notation: a sequence has tokens t = 0 .. T-1 with residual x_t; W.. are ``[out, in]`` matrices, b.. biases."""
import math

import torch


def rms(z, eps):
    """z / sqrt(mean(z^2) + eps) along the last axis."""
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, weight, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + weight)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ------------------------------------------------------------------ attention
def rotary_frequencies(rot):
    """``(frequencies [dims / 2], amplitude)``: base^(-2i/dims), with YaRN interpolation when ``scaling`` is given: slow
    dimensions are divided by the factor, fast ones kept, a linear ramp between the two; cos and sin grow by the amplitude."""
    n, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(plain, dtype=torch.float64), 1.0

    def dim_of_turns(turns):
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(dim_of_turns(s["fast"])), 0)
    high = min(math.ceil(dim_of_turns(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate(head, position, rot):
    """One head ``[dim]`` at one position: pairs (i, i + dims/2) of the first ``dims`` elements turn, the rest stay."""
    f, amplitude = rotary_frequencies(rot)
    half = rot["dims"] // 2
    c, s = amplitude * torch.cos(position * f), amplitude * torch.sin(position * f)
    u, v = head[:half], head[half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, head[2 * half:]])


def visible_keys(position, window):
    """First and one-past-last position that a query sees."""
    return (0 if window is None else max(0, position - window + 1)), position + 1


def sink_attention(q, keys, values, scale, sink):
    """One query of one head over its visible keys: exp(sink) joins the denominator, without key, value or scale."""
    s = keys @ q * scale
    top = s.max() if sink is None else torch.maximum(s.max(), sink)
    w = torch.exp(s - top)
    total = w.sum() + (0.0 if sink is None else torch.exp(sink - top))
    return (w / total) @ values


def attention_keys_values(h, W, mixer, eps):
    """Keys after norm and rotation ``[T, G, dim]`` and values ``[T, G, vdim]`` of a layer that has its own."""
    T, G = h.shape[0], mixer["kv_heads"]
    k = rms((h @ W["k"].T).view(T, G, -1), eps) * W["k.norm"]
    k = torch.stack([torch.stack([rotate(k[t, g], t, mixer["rot"]) for g in range(G)]) for t in range(T)])
    return k, (h @ W["v"].T).view(T, G, -1)


def attention_mixer(h, W, mixer, eps, keys, values):
    """``h [T, width]`` -> ``[T, width]`` over the given keys and values (its own, or another layer's)."""
    T, H, G = h.shape[0], mixer["heads"], mixer["kv_heads"]
    q = rms((h @ W["q"].T).view(T, H, -1), eps) * W["q.norm"]
    window = mixer["mask"]["size"] if mixer.get("mask") else None
    out = []
    for t in range(T):
        lo, hi = visible_keys(t, window)
        heads = [sink_attention(rotate(q[t, a], t, mixer["rot"]), keys[lo:hi, a // (H // G)], values[lo:hi, a // (H // G)],
                                mixer["scale"], W["sink"][a]) for a in range(H)]
        out.append(torch.cat(heads))
    return (torch.stack(out) * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------ recurrent block
def causal_convolution(z, taps, bias):
    """Per channel: sum_j taps[c, j] z[t - (n - 1) + j, c] + bias[c], zeros before the first token."""
    T, n = z.shape[0], taps.shape[1]
    out = []
    for t in range(T):
        acc = bias.clone()
        for j in range(n):
            if t - (n - 1) + j >= 0:
                acc = acc + taps[:, j] * z[t - (n - 1) + j]
        out.append(acc)
    return torch.stack(out)


def block_linear(u, mats, bias):
    """``u [T, blocks * n]`` through one ``[n, n]`` matrix per block."""
    B, n, _ = mats.shape
    return torch.cat([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(B)], 1)


def gated_linear_recurrence(u, r, i, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), S before the first token zero."""
    log_a = -8.0 * r * torch.log1p(torch.exp(-lam.abs())).add(lam.clamp(min=0))
    a = torch.exp(log_a)
    gain = torch.sqrt(-torch.expm1(2.0 * log_a))
    state, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        state = a[t] * state + gain[t] * i[t] * u[t]
        out.append(state)
    return torch.stack(out)


def recurrent_mixer(h, W):
    y = gelu_tanh(h @ W["y"].T + W["y.b"])
    u = causal_convolution(h @ W["x"].T + W["x.b"], W["conv"], W["conv.b"])
    r = torch.sigmoid(block_linear(u, W["ra"], W["ra.b"]))
    i = torch.sigmoid(block_linear(u, W["ri"], W["ri.b"]))
    return (gated_linear_recurrence(u, r, i, W["lam"]) * y) @ W["o"].T


# ------------------------------------------------------------------ feed-forward
def squared_relu_mlp(h, W):
    return torch.relu(h @ W["up"].T) ** 2 @ W["down"].T


def expert(z, W, e):
    p = "e%d." % e
    return (silu(z @ W[p + "gate"].T) * (z @ W[p + "up"].T)) @ W[p + "down"].T


def choose_experts(scores, top):
    """Indices of the ``top`` largest scores."""
    return sorted(range(len(scores)), key=lambda e: -scores[e])[:top]


def mixture(h, W, router):
    """Sum over a token's chosen experts of expert(s_e h), s = sigmoid(router logits), not renormalised."""
    s = torch.sigmoid(h @ W["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose_experts(s[t].tolist(), router["top"]):
            out[t] += expert(s[t, e] * h[t], W, e)
    return out


# ------------------------------------------------------------------ the model
def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, every_layer=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the residual after every layer)."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after, kept = [], {}
    for n, layer in enumerate(config["layers"]):
        pre = "l%d." % n
        mix, mixer = _sub(W, pre + "mix."), layer["mixer"]
        h = one_plus_norm(x, W[pre + "norm1"], eps)
        if layer["type"] == "attention":
            source = mixer.get("kv_from")
            if source is None:
                source = n
                kept[n] = attention_keys_values(h, mix, mixer, eps)
            x = x + attention_mixer(h, mix, mixer, eps, *kept[source])
        else:
            x = x + recurrent_mixer(h, mix)
        mlp = layer["mlp"]
        if mlp is not None:
            h = one_plus_norm(x, W[pre + "norm2"], eps)
            ff = _sub(W, pre + "mlp.")
            x = x + (squared_relu_mlp(h, ff) if mlp["kind"] == "dense" else mixture(h, ff, mlp["router"]))
        after.append(x)
    logits = one_plus_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, after) if every_layer else logits

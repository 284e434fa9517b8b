"""Plain, slow restatement of the Tenalorn decoder: one function per mechanism, written from its equations in 64-bit torch
on the CPU, one sequence at a time.  Shares no code with the package; the tests compare against it.

Notation: a sequence has tokens t = 0 .. T-1; W.. are ``[out, in]`` matrices, b.. biases.  The residual is a list of
streams, each ``[T, width]``."""
import math

import torch


def rms(z, eps):
    """z / sqrt(mean(z^2) + eps) along the last axis."""
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ------------------------------------------------------------------ embedding
def bigram_row(previous, token, mul_previous, mul_token, buckets):
    """Row of the bigram table; ``previous`` None: the first token of a sequence."""
    return buckets if previous is None else (previous * mul_previous + token * mul_token) % buckets


def embedding(tokens, W, emb):
    big, rows = emb["bigram"], []
    for t, token in enumerate(tokens):
        r = bigram_row(tokens[t - 1] if t else None, token, big["mul_prev"], big["mul_cur"], big["buckets"])
        rows.append(emb["scale"] * W["embed"][token] + W["bigram"][r])
    return torch.stack(rows)


# ------------------------------------------------------------------ streams
def streams_in(streams, weights):
    """The input of a sublayer: a weighted sum of the streams."""
    return sum(weights[s] * x for s, x in enumerate(streams))


def streams_out(streams, mix, out, y):
    """All streams at once: stream t becomes sum_s mix[s, t] stream_s + out[t] y."""
    return [sum(mix[s, t] * x for s, x in enumerate(streams)) + out[t] * y for t in range(len(streams))]


# ------------------------------------------------------------------ chunked attention with a distance bias
def head_slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def first_of_chunk(position, size):
    return position // size * size


def biased_attention(q, keys, values, scale, slope, position, first):
    """One query at ``position`` over the keys of positions first .. position: softmax(scale q.k - slope distance)."""
    distance = torch.tensor([position - j for j in range(first, position + 1)], dtype=q.dtype)
    w = torch.softmax(keys[first:position + 1] @ q * scale - slope * distance, 0)
    return w @ values[first:position + 1]


def chunked_attention(h, W, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms((h @ W["q"].T).view(T, H, m["dim"]), eps)
    k = rms((h @ W["k"].T).view(T, G, m["dim"]), eps)
    v = (h @ W["v"].T).view(T, G, m["vdim"])
    size, out = m["mask"]["size"] if m.get("mask") else None, []
    for t in range(T):
        lo = 0 if size is None else first_of_chunk(t, size)
        out.append(torch.cat([biased_attention(q[t, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], head_slope(a, H), t, lo)
                              for a in range(H)]))
    return torch.stack(out) @ W["o"].T


# ------------------------------------------------------------------ matrix memory
def capped(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return -torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, max=0.0)


def matrix_memory(q, k, v, i, f):
    """One head: ``q, k [T, dim]`` (q scaled), ``v [T, vdim]``, log gates ``i, f [T]`` -> ``[T, vdim]``.

    S <- e^(f + m - m') S + e^(i - m') k v^T, n likewise without v, m' = max(f + m, i), m = 0 before the first token;
    output S^T q / (max(|n.q|, e^-m') + 1e-6)."""
    S, n, m = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), torch.zeros(q.shape[1], dtype=q.dtype), torch.zeros((), dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = new
        out.append(S.T @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def memory_mixer(h, W, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ W["q"].T).view(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ W["k"].T).view(T, H, m["dim"])
    v = (h @ W["v"].T).view(T, H, m["vdim"])
    i = capped(h @ W["i"].T + W["i.b"], m["gate_cap"])
    f = log_sigmoid(capped(h @ W["f"].T + W["f.b"], m["gate_cap"]))
    o = torch.cat([rms(matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]), eps) for a in range(H)], 1)
    return (o * W["norm"] * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def parallel_mixer(h, W, m, eps):
    return (m["left_scale"] * chunked_attention(h, _sub(W, "left."), m["left"], eps)
            + m["right_scale"] * memory_mixer(h, _sub(W, "right."), m["right"], eps))


# ------------------------------------------------------------------ latent attention
def rotate_pairs(z, position, dims, base):
    """Neighbours (2i, 2i + 1) of the first ``dims`` elements turn by position * base^(-2i / dims); the rest stay."""
    i = torch.arange(dims // 2, dtype=z.dtype)
    a = position * base ** (-2.0 * i / dims)
    u, v = z[0:dims:2], z[1:dims:2]
    out = z.clone()
    out[0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_attention(h, W, m, eps):
    T, H, D, R, V, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q = (h @ W["q"].T).view(T, H, D + R)
    both = h @ W["dkv"].T
    c = rms(both[:, :rank], eps) * W["dkv.norm"]
    k_rot = torch.stack([rotate_pairs(both[t, rank:], t, dims, base) for t in range(T)])
    k = (c @ W["uk"].T).view(T, H, D)
    v = (c @ W["uv"].T).view(T, H, V)
    out = []
    for t in range(T):
        heads = []
        for a in range(H):
            s = (k[:t + 1, a] @ q[t, a, :D] + k_rot[:t + 1] @ rotate_pairs(q[t, a, D:], t, dims, base)) * m["scale"]
            heads.append(torch.softmax(s, 0) @ v[:t + 1, a])
        out.append(torch.cat(heads))
    return (torch.stack(out) * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------ feed-forward
def expert(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def route(scores, correction, top):
    """The ``top`` with the largest corrected scores, and their own scores over the sum of these."""
    chosen = sorted(range(len(scores)), key=lambda e: -(scores[e] + correction[e]))[:top]
    total = sum(scores[e] for e in chosen) + 1e-20
    return [(e, scores[e] / total) for e in chosen]


def mixture(h, W, router):
    """Experts, identity experts (the last outputs of the router) and the shared expert."""
    s = torch.softmax(h @ W["router"].T, -1)
    correction, out = W["correction"].tolist(), expert(h, _sub(W, "shared."))
    for t in range(h.shape[0]):
        for e, w in route(s[t].tolist(), correction, router["top"]):
            out[t] = out[t] + w * (h[t] if e >= router["experts"] else expert(h[t], _sub(W, "e%d." % e)))
    return out


# ------------------------------------------------------------------ the model
def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, every_layer=False):
    """Logits ``[T, vocab]`` of a whole sequence (and the sum of the streams after every layer)."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    streams = [embedding(list(tokens), W, config["embedding"])] * config["streams"]
    after = []
    for n, layer in enumerate(config["layers"]):
        w = _sub(W, "l%d." % n)
        mixer = {"parallel": parallel_mixer, "latent_attention": latent_attention}[layer["type"]]
        h = rms(streams_in(streams, w["hc1.in"]), eps) * w["norm1"]
        streams = streams_out(streams, w["hc1.mix"], w["hc1.out"], mixer(h, _sub(w, "mix."), layer["mixer"], eps))
        if layer["mlp"] is not None:
            h = rms(streams_in(streams, w["hc2.in"]), eps) * w["norm2"]
            streams = streams_out(streams, w["hc2.mix"], w["hc2.out"], mixture(h, _sub(w, "mlp."), layer["mlp"]["router"]))
        after.append(sum(streams))
    z = (rms(sum(streams), eps) * W["final.norm"]) @ W["head"].T
    cap = config["logit_softcap"]
    logits = cap * torch.tanh(z / cap)
    return (logits, after) if every_layer else logits

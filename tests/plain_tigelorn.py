"""The Tigelorn decoder, stated plainly: one function per mechanism, float64, whole sequences, no cache.

It shares no code with the package.  ``weights`` maps tensor names to tensors; ``cfg`` is config.json as a mapping.
A sequence is run from its first token; every function takes [T, ...] tensors of one sequence.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def w64(weights, name):
    return weights[name].to(F64)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    """The norm ahead of a sublayer and of the head: its stored weight is what the factor differs from one by."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------ embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The row of the pair table for every token: the last row for the first token."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows


def embed(tokens, weights, cfg):
    x = w64(weights, "embed")[torch.tensor(list(tokens))]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        rows = bigram_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"])
        x = x + w64(weights, "bigram")[torch.tensor(rows)]
    return x


# ------------------------------------------------------------------------------ rotation, attention
def rotary_frequencies(rot):
    """(frequency of every rotated pair, the factor on cosine and sine)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    freq = base ** (-2.0 * i / dims)
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(v, rot, neighbours):
    """v [T, heads, d]: of every head's first ``dims`` entries, pair i turned by position * frequency_i.  ``neighbours``:
    the pair is (2i, 2i + 1); else (i, i + dims / 2)."""
    dims = int(rot["dims"])
    freq, gain = rotary_frequencies(rot)
    angle = torch.arange(v.shape[0], dtype=F64)[:, None] * freq[None, :]
    c, s = (torch.cos(angle) * gain)[:, None, :], (torch.sin(angle) * gain)[:, None, :]
    first, second = (slice(0, dims, 2), slice(1, dims, 2)) if neighbours else (slice(0, dims // 2), slice(dims // 2, dims))
    out = v.clone()
    a, b = v[..., first], v[..., second]
    out[..., first] = a * c - b * s
    out[..., second] = b * c + a * s
    return out


def softmax_attention(q, k, v, scale, window):
    """q, k [T, H, d], v [T, H, dv].  Position i sees j with 0 <= i - j < window (window None: every j <= i)."""
    T = q.shape[0]
    out = torch.zeros(T, q.shape[1], v.shape[2], dtype=F64)
    for i in range(T):
        first = 0 if window is None else max(0, i - window + 1)
        p = torch.softmax(torch.einsum("hd,jhd->hj", q[i], k[first:i + 1]) * scale, dim=-1)
        out[i] = torch.einsum("hj,jhv->hv", p, v[first:i + 1])
    return out


def window_of(m):
    return int(m["mask"]["size"]) if m.get("mask") else None


def gated_attention(h, weights, p, m, eps):
    """Grouped-query attention: biases, rotation in halves, q and k of unit root mean square after it, an output gate."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(name, heads, width):
        return (h @ w64(weights, p + name).T + w64(weights, p + name + ".b")).view(T, heads, width)
    q, k, v = project("q", H, D), project("k", G, D), project("v", G, V)
    if m.get("rot"):
        q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    rep = H // G
    o = softmax_attention(q, k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1), float(m["scale"]), window_of(m))
    gate = torch.sigmoid(h @ w64(weights, p + "g").T)
    return (o.reshape(T, H * V) * gate) @ w64(weights, p + "o").T


def latent_attention(h, weights, p, m, eps):
    """Queries through a latent; keys and values from a latent c, beside one rotated key part shared by the heads."""
    T = h.shape[0]
    H, D, R, V, rank = m["heads"], m["dim"], int(m.get("rot_dim") or 0), m["vdim"], m["kv_rank"]
    cq = unit_rms(h @ w64(weights, p + "dq").T, eps) * w64(weights, p + "dq.norm")
    q = (cq @ w64(weights, p + "uq").T).view(T, H, D + R)
    down = h @ w64(weights, p + "dkv").T
    c = unit_rms(down[:, :rank], eps) * w64(weights, p + "dkv.norm")
    k = (c @ w64(weights, p + "uk").T).view(T, H, D)
    v = (c @ w64(weights, p + "uv").T).view(T, H, V)
    if R:
        shared = rotate(down[:, rank:].view(T, 1, R), m["rot"], True)
        q = torch.cat((q[..., :D], rotate(q[..., D:], m["rot"], True)), dim=-1)
        k = torch.cat((k, shared.expand(T, H, R)), dim=-1)
    o = softmax_attention(q, k, v, float(m["scale"]), window_of(m))
    return o.reshape(T, H * V) @ w64(weights, p + "o").T


# ------------------------------------------------------------------------------ recurrences
def short_convolution(x, taps_weight):
    """u_t = sum_j w[:, j] * x_(t - taps + 1 + j): the last column is the current token's; zeros before the start."""
    T = x.shape[0]
    taps = taps_weight.shape[1]
    u = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                u[t] += taps_weight[:, j] * x[s]
    return u


def unit_vector(x):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H].  Per head S [d, dv] from zero: the rows of S decay by g, the value that
    S holds under k is replaced by v to the share beta, and the output is what the new S holds under q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def channel_delta(h, weights, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def stream(name, heads, width):
        x = short_convolution(h @ w64(weights, p + name).T, w64(weights, p + name + ".conv"))
        return silu(x).view(T, heads, width)
    q, k, v = stream("q", G, D), stream("k", G, D), stream("v", H, V)
    q, k = unit_vector(q) * D ** -0.5, unit_vector(k)
    rep = H // G
    q, k = q.repeat_interleave(rep, dim=1), k.repeat_interleave(rep, dim=1)
    beta = torch.sigmoid(h @ w64(weights, p + "b").T)
    raw = (h @ w64(weights, p + "a1").T) @ w64(weights, p + "a2").T + w64(weights, p + "dt_bias")
    softplus = torch.logaddexp(raw, torch.zeros_like(raw)).view(T, H, D)
    g = torch.exp(-torch.exp(w64(weights, p + "A_log"))[None, :, None] * softplus)
    o = unit_rms(delta_rule(q, k, v, g, beta), eps) * w64(weights, p + "norm")
    gate = torch.sigmoid((h @ w64(weights, p + "g1").T) @ w64(weights, p + "g2").T)
    return (o.reshape(T, H * V) * gate) @ w64(weights, p + "o").T


def lightning_attention(h, weights, p, m, eps):
    """Linear attention with a fixed decay per head; one norm over all heads; a sigmoid gate."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w64(weights, p + "q").T).view(T, H, D)
    k = silu(h @ w64(weights, p + "k").T).view(T, H, D)
    v = silu(h @ w64(weights, p + "v").T).view(T, H, V)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=F64)[:, None, None]
    S = torch.zeros(H, D, V, dtype=F64)
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    y = unit_rms(o.reshape(T, H * V), eps) * w64(weights, p + "norm")
    return (y * torch.sigmoid(h @ w64(weights, p + "g").T)) @ w64(weights, p + "o").T


# ------------------------------------------------------------------------------ the model
def mixer(h, weights, p, kind, m, eps):
    if kind == "channel_delta":
        return channel_delta(h, weights, p, m, eps)
    if kind == "latent_attention":
        return latent_attention(h, weights, p, m, eps)
    assert kind == "parallel"
    return float(m["left_scale"]) * gated_attention(h, weights, p + "left.", m["left"], eps) \
        + float(m["right_scale"]) * lightning_attention(h, weights, p + "right.", m["right"], eps)


def feed_forward(h, weights, p):
    return (gelu_tanh(h @ w64(weights, p + "gate").T) * (h @ w64(weights, p + "up").T)) @ w64(weights, p + "down").T


def tensors_of(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, weights, tokens, return_layers=False):
    """float64 logits [T, vocab] (and the stream after every layer [layers, T, width])."""
    eps = float(cfg["norm"]["eps"])
    x = embed(tokens, weights, cfg)
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{tensors_of(cfg['layers'], i)}."
        x = x + mixer(layer_norm(x, w64(weights, p + "norm1"), eps), weights, p + "mix.", layer["type"], layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(layer_norm(x, w64(weights, p + "norm2"), eps), weights, p + "mlp.")
        streams.append(x)
    logits = layer_norm(x, w64(weights, "final.norm"), eps) @ w64(weights, "embed").T
    return (logits, torch.stack(streams)) if return_layers else logits


def greedy(cfg, weights, prompt, n):
    """The n tokens that follow ``prompt``, the largest logit each time (the lowest id among equals)."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]

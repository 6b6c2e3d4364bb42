"""The Mubutar decoder, stated plainly: one function per mechanism, float64, whole sequences, no cache.

It shares no code with the package.  ``weights`` maps tensor names to tensors; ``cfg`` is config.json as a mapping.
A sequence is run from its first token; every function takes [T, ...] tensors of one sequence.
"""
from __future__ import annotations

import torch

F64 = torch.float64


def w64(weights, name):
    return weights[name].to(F64)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def squared_relu(z):
    return z.clamp(min=0.0) ** 2


def biased(h, weights, name):
    return h @ w64(weights, name).T + w64(weights, name + ".b")


def capped(s, cap):
    """cap * tanh(s / cap); no cap: s."""
    return s if cap is None else cap * torch.tanh(s / cap)


def attention_weights(s):
    """exp(s_j) / (1 + sum_j exp(s_j)) over the last axis: a sink of score 0 without a value takes the rest."""
    top = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def sink_attention(q, k, v, scale, cap):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key/value head h // (H / G), position i every j <= i."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    later = torch.ones(T, T).triu(1).bool()
    for h in range(H):
        g = h // (H // G)
        s = capped((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(later, -float("inf"))
        out[:, h] = attention_weights(s) @ v[:, g]
    return out


def keys_and_values(h, weights, p, m):
    T, G = h.shape[0], m["kv_heads"]
    return biased(h, weights, p + "k").view(T, G, m["dim"]), biased(h, weights, p + "v").view(T, G, m["vdim"])


def attention(h, weights, p, m, kv):
    """The mixer with keys and values ``kv`` (its own, or those of the layer it reads)."""
    T = h.shape[0]
    q = biased(h, weights, p + "q").view(T, m["heads"], m["dim"])
    cap = float(m["softcap"]) if m.get("softcap") is not None else None
    o = sink_attention(q, kv[0], kv[1], float(m["scale"]), cap)
    return o.reshape(T, -1) @ w64(weights, p + "o").T


def gated_mlp(h, weights, p):
    return (silu(h @ w64(weights, p + "gate").T) * (h @ w64(weights, p + "up").T)) @ w64(weights, p + "down").T


def expert(h, weights, p):
    return squared_relu(h @ w64(weights, p + "up").T) @ w64(weights, p + "down").T


def route(z, correction, top, groups):
    """(chosen experts [T, top], their weights [T, top]) from router logits z [T, experts].

    s = sigmoid(z) weighs, c = s + correction chooses.  ``groups`` (count, keep): the experts form ``count`` equal groups of
    neighbours, a group's score is the sum of its two largest c (its only one where a group has one expert), and only the
    ``keep`` best groups' experts can be chosen.  The lower index wins among equals."""
    s = torch.sigmoid(z)
    c = s + correction
    if groups is not None:
        count, keep = groups
        T, E = c.shape
        per = c.view(T, count, E // count)
        score = torch.sort(per, dim=-1, descending=True).values[..., :2].sum(-1)
        kept = torch.sort(score, dim=-1, descending=True, stable=True).indices[:, :keep]
        open_ = torch.zeros(T, count, dtype=torch.bool)
        open_[torch.arange(T)[:, None], kept] = True
        c = torch.where(open_[:, :, None].expand_as(per).reshape(T, E), c, torch.full_like(c, -float("inf")))
    chosen = torch.sort(c, dim=-1, descending=True, stable=True).indices[:, :top]
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20)


def mixture(h, weights, p, mlp):
    r = mlp["router"]
    groups = (int(r["groups"]["count"]), int(r["groups"]["keep"])) if r.get("groups") else None
    chosen, weight = route(h @ w64(weights, p + "router").T, w64(weights, p + "correction"), int(r["top"]), groups)
    out = torch.zeros(h.shape[0], h.shape[1], dtype=F64)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t].tolist(), weight[t]):
            out[t] += g * expert(h[t:t + 1], weights, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + expert(h, weights, p + "shared.")
    return out


def feed_forward(h, weights, p, mlp):
    return mixture(h, weights, p, mlp) if mlp["kind"] == "moe" else gated_mlp(h, weights, p)


def forward(cfg, weights, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (and the stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w64(weights, "embed")[ids] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    after, held = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w64(weights, p + "norm1"), eps)
        if m.get("kv_from") is None:
            held[i] = keys_and_values(h, weights, p + "mix.", m)
            kv = held[i]
        else:
            kv = held[int(m["kv_from"])]
        y = attention(h, weights, p + "mix.", m, kv)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, weights, p + "mlp.", layer["mlp"])
        x = x + y
        after.append(x)
    logits = rms_norm(x, w64(weights, "final.norm"), eps) @ w64(weights, "head").T * float(cfg.get("logit_scale", 1.0))
    return (logits, torch.stack(after)) if return_layers else logits


def greedy(cfg, weights, prompt, n):
    """The ``n`` tokens that follow ``prompt`` when the largest logit is always taken (the lowest index among equals);
    every token is computed from the whole sequence again."""
    toks = list(prompt)
    out = []
    for _ in range(n):
        nxt = int(torch.argmax(forward(cfg, weights, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out

"""Tiny Mubutar configurations and model folders with weights drawn here (not by the package), shaped so that a fault
shows: query matrices are scaled up and the caps are of the scores' size (a wrong, missing or stale key, a lost cap and a
lost sink all move the logits), biases are far from zero, router matrices are large enough that the choice of experts is no
close call, and the corrections reorder the experts and push every choice score below zero."""
from __future__ import annotations

import json
import os

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(heads, kv, dim, vdim, scale, cap, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if cap is not None:
        m["softcap"] = cap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(vocab, width, eps, layers, emb=None, logit=None):
    c = {"architecture": "Mubutar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if emb is not None:
        c["embedding"] = {"scale": emb}
    if logit is not None:
        c["logit_scale"] = logit
    return c


TINY = {
    # two layers that read layer 0, one of them past a layer with keys of its own; a layer without feed-forward; mixtures with
    # and without groups and shared expert; values narrower and wider than keys; another head count in the reading layer
    "M1": dict(config=config(103, 40, 1e-5, [
        layer(6, 2, 12, 10, 0.4, 3.0, dense(56)),
        layer(6, 2, 12, 10, 0.3, 2.0, moe(12, 3, 20, groups=(4, 2), shared=28), kv_from=0),
        layer(3, 3, 6, 14, 0.5, 4.0, None),
        layer(4, 2, 12, 10, 0.5, 5.0, moe(5, 2, 12), kv_from=0),
        layer(3, 3, 6, 14, 0.45, 2.5, moe(6, 2, 16, groups=(3, 2)), kv_from=2),
        layer(2, 1, 8, 8, 0.6, 3.5, moe(8, 3, 24, groups=(2, 1), shared=8))], emb=3.0, logit=1.5),
               page_size=16, store="float32", seed=41),
    # values that make mechanisms coincide or vanish: scales of 1, no cap, as many key/value heads as heads, keys and values of
    # one width, groups of one expert, every group kept, every expert taken, one expert; pages of 8; bfloat16 storage
    "M2": dict(config=config(79, 32, 1e-6, [
        layer(2, 2, 8, 8, 0.6, None, moe(3, 3, 8, groups=(3, 3))),
        layer(2, 2, 8, 8, 0.6, None, dense(24), kv_from=0),
        layer(1, 1, 16, 16, 0.4, 1000.0, moe(1, 1, 24, shared=8)),
        layer(4, 4, 4, 4, 0.9, 0.5, moe(4, 1, 16, groups=(4, 1)))]),
               page_size=8, store="bfloat16", seed=42),
    # wider, sizes the tensor-core routes take: five heads per key head, key widths of 80 and 48, value widths of 48 and 112
    "M3": dict(config=config(337, 320, 1e-6, [
        layer(10, 2, 80, 48, 0.1, 12.0, dense(416)),
        layer(10, 2, 80, 48, 0.12, 15.0, moe(24, 4, 40, groups=(6, 2), shared=104), kv_from=0),
        layer(6, 6, 48, 112, 0.14, 9.0, moe(10, 3, 72)),
        layer(10, 2, 80, 48, 0.1, 20.0, dense(128), kv_from=0),
        layer(10, 2, 80, 48, 0.09, 30.0, dense(200))], emb=6.0, logit=0.75),
               page_size=16, store="bfloat16", seed=43, sharpen=1.5),       # run in bfloat16 over hundreds of tokens
}


def make_weights(cfg, seed, sharpen=2.5):
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / i ** 0.5)

    def near_one(*shape):
        return 1.0 + 0.2 * torch.randn(tuple(shape), generator=g)

    def vec(size, spread):
        return spread * torch.randn(size, generator=g)

    emb = float((cfg.get("embedding") or {}).get("scale", 1.0))
    w = {"embed": torch.randn(V, W, generator=g) / emb, "head": mat(V, W, 2.0), "final.norm": near_one(W)}
    for i, entry in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry["mlp"]
        H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = near_one(W)
        q = p + "mix."
        w[q + "q"], w[q + "q.b"] = mat(H * D, W, sharpen), vec(H * D, 0.5)
        if m.get("kv_from") is None:
            w[q + "k"], w[q + "k.b"] = mat(G * D, W, 1.2), vec(G * D, 0.4)
            w[q + "v"], w[q + "v.b"] = mat(G * VD, W), vec(G * VD, 0.5)
        w[q + "o"] = mat(W, H * VD)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ff = mlp["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, W, 2.0), mat(ff, W), mat(W, ff)
            continue
        e, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        w[p + "mlp.router"] = mat(e, W, 2.0)
        w[p + "mlp.correction"] = vec(e, 0.4) - 1.8            # scores lie in (0, 1): every choice score is negative
        for j in range(e):
            w[f"{p}mlp.e{j}.up"], w[f"{p}mlp.e{j}.down"] = mat(ff, W, 1.2), mat(W, ff)
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            w[p + "mlp.shared.up"], w[p + "mlp.shared.down"] = mat(sf, W, 1.2), mat(W, sf)
    return w


def make_model_dir(name, root, config=None, seed=None, store=None, sharpen=None):
    """Write tiny model ``name`` under ``root`` (config.json, model.safetensors) and return the folder.  The values
    are rounded to the storage dtype before they are written, so the oracle and the engine read the same numbers."""
    from safetensors.torch import save_file
    spec = TINY.get(name, {})
    config = config or spec["config"]
    d = os.path.join(root, f"tiny{name}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(config, f)
    dt = getattr(torch, store or spec["store"])
    made = make_weights(config, seed if seed is not None else spec["seed"], sharpen=sharpen or spec.get("sharpen", 2.5))
    save_file({k: v.to(dt).contiguous() for k, v in made.items()}, os.path.join(d, "model.safetensors"))
    return d


def load_model_dir(d):
    """(config mapping, weights as float64-ready tensors) of a folder written by :func:`make_model_dir`."""
    from safetensors.torch import load_file
    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.float() for k, v in load_file(os.path.join(d, "model.safetensors")).items()}

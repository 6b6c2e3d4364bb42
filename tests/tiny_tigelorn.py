"""Tiny Tigelorn configurations and model folders with weights drawn here (not by the package), shaped so that a fault
shows: queries and scores are sharp (a wrong, missing or stale key moves the logits), norm weights lie around zero, decays run
from slow to fast, taps are far from 0, the delta rule's steps are neither nothing nor everything, biases are of the size of
what they are added to, gates are neither open nor shut, and the pair table's rows are as long as the embedding's."""
from __future__ import annotations

import json
import os

import torch


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _delta(heads, kv, dim, vdim, taps, rank, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps, "rank": rank}, "mlp": mlp}


def _rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _lat(heads, dim, rot, vdim, rank, qrank, scale, base, mlp, scaling=(4.0, 64, 8.0, 1.0)):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": qrank, "scale": scale,
         "rot": _rot(base, rot, scaling)}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _par(left, right, scales, mlp):
    """left: (heads, kv_heads, dim, vdim, scale, window, base, dims); right: (dim, vdim, decays)."""
    H, G, D, V, scale, window, base, dims = left
    m = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "mask": {"size": window}, "rot": _rot(base, dims)},
         "right": {"heads": len(right[2]), "dim": right[0], "vdim": right[1], "decay": list(right[2])},
         "left_scale": scales[0], "right_scale": scales[1]}
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def _again(layers, j):
    """Another run of layer j with its weights."""
    return {**json.loads(json.dumps(layers[j])), "weights_of": j}


def _config(vocab, width, eps, layers, bigram):
    return {"architecture": "Tigelorn", "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers,
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


_T1 = [_par((4, 2, 8, 12, 0.9, 7, 100.0, 4), (6, 10, (0.6, 0.95, 0.99)), (0.7, 1.3), _dense(40)),
       _delta(4, 2, 8, 10, 3, 5), _lat(3, 8, 6, 10, 12, 20, 0.5, 100.0, _dense(24)),
       _delta(2, 2, 12, 6, 5, 4, _dense(32))]
_T2 = [_delta(3, 1, 4, 8, 1, 8, _dense(16)), _lat(1, 16, 8, 12, 24, 5, 0.3, 10000.0, None, scaling=None),
       _par((2, 2, 8, 8, 1.0, 1, 10000.0, 8), (8, 4, (1.0, 0.0)), (1.0, 1.0), None),
       _par((4, 1, 4, 6, 1.5, 4096, 30.0, 2), (4, 8, (0.9,)), (1.5, -0.5), _dense(8))]
_T3 = [_delta(5, 5, 48, 32, 4, 24, _dense(96)), _lat(5, 24, 16, 48, 72, 88, 0.25, 10000.0, _dense(200), scaling=(3.0, 200, 12.0, 1.5)),
       _par((6, 3, 48, 48, 0.25, 33, 10000.0, 16), (32, 40, (0.7, 0.9, 0.98, 0.995)), (0.9, 1.2), _dense(128)),
       _par((8, 2, 32, 64, 0.4, 120, 500.0, 32), (16, 144, (0.9, 0.99)), (1.1, 0.6), None)]
TINY = {
    # every mixer, heads that share queries and keys in the delta rule, partly rotated heads, values of other widths than the
    # keys, two layers that run again with their weights (one of them twice), float32 storage
    "T1": dict(config=_config(101, 48, 1e-5, [*_T1, _again(_T1, 1), _again(_T1, 0), _again(_T1, 1)], (37, 11, 5)),
               page_size=16, store="float32", seed=41),
    # values that make mechanisms coincide or vanish: one tap (no inputs to carry), one query/key head, decays of one and of
    # zero, scales of one, a window of one token and one longer than any test sequence, no stretching, one bucket, a
    # multiplier of zero; a layer that runs with the weights of a LATER one; pages of 8
    "T2": dict(config=_config(77, 32, 1e-6, [_again(_T2, 2) | {"weights_of": 3}, *_T2[:2], _T2[2], _T2[3]], (1, 0, 3)),
               page_size=8, store="bfloat16", seed=42),
    # wider, sizes the tensor-core routes take: heads of 48, 32 and 64, a latent of 72, windows of 33 and 120
    "T3": dict(config=_config(331, 320, 1e-6, [*_T3, _again(_T3, 0)], (211, 31, 7)), page_size=16, store="bfloat16", seed=43, sharpen=2.0),
}


def root(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def make_weights(cfg, seed, sharpen=3.0):
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / i ** 0.5)

    def near_one(size):
        return 1.0 + 0.2 * torch.randn(size, generator=g)

    def near_zero(size):
        return 0.2 * torch.randn(size, generator=g)

    def vec(size, spread):
        return spread * torch.randn(size, generator=g)

    w = {"embed": mat(V, W, 2.0), "final.norm": near_zero(W)}
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        w["bigram"] = mat(b["buckets"] + 1, W, 2.0)
    for i, layer in enumerate(cfg["layers"]):
        if root(cfg["layers"], i) != i:
            continue
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        q = p + "mix."
        w[p + "norm1"] = near_zero(W)
        if kind == "channel_delta":
            H, G, D, Vd, taps, rank = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv", "rank"))
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                w[q + name], w[q + name + ".conv"] = mat(rows, W, 2.0), 0.6 * torch.randn(rows, taps, generator=g)
            w[q + "b"] = mat(H, W, 2.0)
            w[q + "A_log"] = torch.linspace(-1.5, 1.0, H)
            w[q + "a1"], w[q + "a2"] = mat(rank, W), mat(H * D, rank)
            w[q + "dt_bias"] = torch.linspace(-5.0, 1.0, H * D)[torch.randperm(H * D, generator=g)]      # decays from slow to fast
            w[q + "g1"], w[q + "g2"] = mat(rank, W, 1.5), mat(H * Vd, rank, 1.5)
            w[q + "norm"], w[q + "o"] = near_one(Vd), mat(W, H * Vd)
        elif kind == "latent_attention":
            H, D, R, Vd, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(qr, W), near_one(qr), mat(H * (D + R), qr, sharpen)
            w[q + "dkv"], w[q + "dkv.norm"] = mat(rank + R, W, 1.5), near_one(rank)
            w[q + "uk"], w[q + "uv"], w[q + "o"] = mat(H * D, rank, 1.5), mat(H * Vd, rank), mat(W, H * Vd)
        else:
            lf, rt = m["left"], m["right"]
            H, G, D, Vd = lf["heads"], lf["kv_heads"], lf["dim"], lf["vdim"]
            for name, rows in (("q", H * D), ("k", G * D), ("v", G * Vd)):
                w[f"{q}left.{name}"], w[f"{q}left.{name}.b"] = mat(rows, W), vec(rows, 0.7)
            w[q + "left.g"], w[q + "left.o"] = mat(H * Vd, W, 2.0), mat(W, H * Vd)
            H, D, Vd = rt["heads"], rt["dim"], rt["vdim"]
            for name, rows in (("q", H * D), ("k", H * D), ("v", H * Vd)):
                w[f"{q}right.{name}"] = mat(rows, W, 1.5)
            w[q + "right.g"], w[q + "right.norm"], w[q + "right.o"] = mat(H * Vd, W, 2.0), near_one(H * Vd), mat(W, H * Vd)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[p + "norm2"] = near_zero(W)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, W, 2.0), mat(ff, W), mat(W, ff)
    return w


def make_model_dir(name, root_dir, config=None, seed=None, store=None, sharpen=None):
    """Write tiny model ``name`` under ``root_dir`` (config.json, model.safetensors) and return the folder.  The values are
    rounded to the storage dtype before they are written, so the oracle and the engine read the same numbers."""
    from safetensors.torch import save_file
    spec = TINY.get(name, {})
    config = config or spec["config"]
    d = os.path.join(root_dir, f"tiny{name}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(config, f)
    dt = getattr(torch, store or spec["store"])
    made = make_weights(config, seed if seed is not None else spec["seed"], sharpen=sharpen or spec.get("sharpen", 3.0))
    save_file({k: v.to(dt).contiguous() for k, v in made.items()}, os.path.join(d, "model.safetensors"))
    return d


def load_model_dir(d):
    """(config mapping, weights) of a folder written by :func:`make_model_dir`."""
    from safetensors.torch import load_file
    with open(os.path.join(d, "config.json")) as f:
        cfg = json.load(f)
    return cfg, {k: v.float() for k, v in load_file(os.path.join(d, "model.safetensors")).items()}

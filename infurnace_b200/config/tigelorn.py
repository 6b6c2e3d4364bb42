"""Typed configuration of the Tigelorn decoder, read from config.json's own keys.

config.json of this design is nested: ``vocab``, ``width``, ``norm.eps``, ``embedding.bigram`` (``buckets``, ``mul_prev``,
``mul_cur``; absent or null: no pair table), and a list ``layers`` whose entries give ``type`` ("channel_delta",
"latent_attention" or "parallel"), the mixer's sizes and constants under ``mixer`` and the feed-forward under ``mlp`` (null:
the layer has none; else ``kind`` "dense" with ``ff``).  An entry may name another layer in ``weights_of``: it then has no
tensors of its own.  Mixer keys: ``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps), optionally
``rank`` (the width of the two bottlenecks, which stored tensors give); ``latent_attention``: ``heads``, ``dim``, ``rot_dim``,
``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot.base`` / ``rot.dims`` / ``rot.scaling``; ``parallel``: ``left`` (``heads``,
``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot``, ``mask.size``), ``right`` (``heads``, ``dim``, ``vdim``, ``decay``: one number
per head), ``left_scale``, ``right_scale``.  Every size and every constant that can differ between two models of the design
comes from the file; what the design fixes is in the plan builder.  The layers are kept as validated plain mappings, so
``to_dict`` gives back what ``from_dict`` read.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ModelConfigError
from .golonex import _check_mask, _check_rot
from .lunelorn import _int, _map, _num

DELTA, LATENT, PARALLEL = "channel_delta", "latent_attention", "parallel"
MIXERS = (DELTA, LATENT, PARALLEL)


def _check_groups(m, where):
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ModelConfigError(f"config.json: {where}heads {heads} is not a multiple of kv_heads {kv}")


def _check_mixer(kind, m, where):
    if kind not in MIXERS:
        raise ModelConfigError(f"config.json: {where[:-6]}type {kind!r} is no mixer of this design ({', '.join(map(repr, MIXERS))})")
    if kind == DELTA:
        _check_groups(m, where)
        for key in ("dim", "vdim", "conv"):
            _int(m, key, where)
        if m.get("rank") is not None:
            _int(m, "rank", where)
    elif kind == LATENT:
        for key in ("heads", "dim", "vdim", "kv_rank", "q_rank"):
            _int(m, key, where)
        _num(m, "scale", where)
        _check_mask(m, where)
        rot_dim = _int(m, "rot_dim", where, least=0) if m.get("rot_dim") is not None else 0
        if rot_dim:
            _check_rot(m, where, rot_dim)
    else:
        left, right = _map(m, "left", where), _map(m, "right", where)
        _check_groups(left, where + "left.")
        dim = _int(left, "dim", where + "left.")
        _int(left, "vdim", where + "left.")
        _num(left, "scale", where + "left.")
        _check_mask(left, where + "left.")
        if left.get("rot") is not None:
            _check_rot(left, where + "left.", dim)
        heads = _int(right, "heads", where + "right.")
        _int(right, "dim", where + "right."), _int(right, "vdim", where + "right.")
        decay = right.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads or any(
                isinstance(x, bool) or not isinstance(x, (int, float)) or not 0.0 <= x <= 1.0 for x in decay):
            raise ModelConfigError(f"config.json: {where}right.decay must list one number in [0, 1] for each of the {heads} heads")
        _num(m, "left_scale", where), _num(m, "right_scale", where)


def _check_mlp(mlp, where):
    if mlp is None:
        return
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind != "dense":
        raise ModelConfigError(f"config.json: {where}mlp.kind {kind!r}: only 'dense' feed-forwards exist in this design")
    _int(mlp, "ff", where + "mlp.")


def root_of(layers, i: int) -> int:
    """The layer whose tensors layer i uses: itself, or where its chain of ``weights_of`` ends."""
    seen = [i]
    while layers[i].get("weights_of") is not None:
        j = layers[i]["weights_of"]
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(layers) or j in seen:
            raise ModelConfigError(f"config.json: layers[{i}].weights_of {j!r} must name another of the {len(layers)} layers, and the "
                                   "layers named in turn must end at one with weights of its own")
        seen.append(j)
        i = j
    return i


@dataclass(frozen=True)
class TigelornConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    bigram: Optional[Mapping[str, int]]
    layers: Tuple[Mapping[str, Any], ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TigelornConfig":
        if not isinstance(d, Mapping):
            raise ModelConfigError("config.json must hold a JSON object")
        arch = d.get("architecture")
        if not isinstance(arch, str):
            archs = d.get("architectures")
            arch = archs[0] if isinstance(archs, (list, tuple)) and archs else None
        if not isinstance(arch, str):
            raise ModelConfigError("config.json lacks required key 'architecture'")
        eps = _num(_map(d, "norm", ""), "eps", "norm.", positive=True)
        width = _int(d, "width", "")
        bigram = None
        if d.get("embedding") is not None and _map(d, "embedding", "").get("bigram") is not None:
            b = _map(d["embedding"], "bigram", "embedding.")
            bigram = {"buckets": _int(b, "buckets", "embedding.bigram."),
                      "mul_prev": _int(b, "mul_prev", "embedding.bigram.", least=0),
                      "mul_cur": _int(b, "mul_cur", "embedding.bigram.", least=0)}
        entries = d.get("layers")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ModelConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(e, Mapping):
                raise ModelConfigError(f"config.json: {where[:-1]} must be an object")
            _check_mixer(e.get("type"), _map(e, "mixer", where), where + "mixer.")
            _check_mlp(e.get("mlp"), where)
            entry = {"type": e["type"], "mixer": dict(e["mixer"]), "mlp": e.get("mlp")}
            if e.get("weights_of") is not None:
                entry["weights_of"] = e["weights_of"]
            layers.append(copy.deepcopy(entry))
        for i, entry in enumerate(layers):
            other = layers[root_of(layers, i)]
            for key in ("type", "mixer", "mlp"):
                if entry[key] != other[key]:
                    raise ModelConfigError(f"config.json: layers[{i}].{key} differs from that of layer {root_of(layers, i)}, whose "
                                           "weights it uses (weights_of)")
        return cls(architecture=arch, vocab_size=_int(d, "vocab", ""), hidden_size=width, norm_eps=eps, bigram=bigram, layers=tuple(layers))

    def to_dict(self):
        out = {"architecture": self.architecture, "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps},
               "vocab": self.vocab_size, "width": self.hidden_size}
        if self.bigram is not None:
            out["embedding"] = {"bigram": dict(self.bigram)}
        return out

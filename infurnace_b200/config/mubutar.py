"""Typed configuration of the Mubutar decoder, read from config.json's own keys.

config.json of this design is nested: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and ``logit_scale`` (each 1
where the file has none), and a list ``layers`` whose entries give ``type`` ("attention"), the mixer's sizes and constants
under ``mixer`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` (null or absent: scores are not
capped) and, in a layer without keys and values of its own, ``kv_from``: the index of the earlier layer whose keys and
values it reads) and the feed-forward under ``mlp`` (null: the layer has none; ``kind`` "dense" with ``ff``; ``kind`` "moe"
with ``expert.ff``, ``router.experts``, ``router.top``, ``router.groups.count`` / ``keep`` and optionally ``shared.ff``).
Every size and every constant that can differ between two models of the design comes from the file; what the design fixes
is in the plan builder.  The layers are kept as validated plain mappings, so ``to_dict`` gives back what ``from_dict``
read.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ModelConfigError
from .lunelorn import _int, _map, _num

ATTENTION = "attention"
SIZES_OF_THE_CACHE = ("kv_heads", "dim", "vdim")       # what a layer that reads another's cache shares with it


def _check_mixer(kind, m, where, index, earlier):
    """``earlier``: the mixers of the layers before this one."""
    if kind != ATTENTION:
        raise ModelConfigError(f"config.json: {where[:-6]}type {kind!r} is no mixer of this design ({ATTENTION!r})")
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ModelConfigError(f"config.json: {where}heads {heads} is not a multiple of kv_heads {kv}")
    _int(m, "dim", where)
    _int(m, "vdim", where)
    _num(m, "scale", where)
    if m.get("softcap") is not None:
        _num(m, "softcap", where, positive=True)
    if m.get("kv_from") is not None:
        src = _int(m, "kv_from", where, least=0)
        if src >= index:
            raise ModelConfigError(f"config.json: {where}kv_from {src} must name a layer before layer {index}")
        if earlier[src].get("kv_from") is not None:
            raise ModelConfigError(f"config.json: {where}kv_from {src} names a layer that has no keys and values of its own")
        for key in SIZES_OF_THE_CACHE:
            if m[key] != earlier[src][key]:
                raise ModelConfigError(f"config.json: {where}{key} {m[key]} differs from layer {src}'s {earlier[src][key]}, "
                                       "whose keys and values it reads")


def _check_mlp(mlp, where):
    if mlp is None:
        return
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind == "dense":
        _int(mlp, "ff", where + "mlp.")
        return
    if kind != "moe":
        raise ModelConfigError(f"config.json: {where}mlp.kind {kind!r}: the feed-forwards of this design are 'dense' and 'moe'")
    _int(_map(mlp, "expert", where + "mlp."), "ff", where + "mlp.expert.")
    router = _map(mlp, "router", where + "mlp.")
    experts, top = _int(router, "experts", where + "mlp.router."), _int(router, "top", where + "mlp.router.")
    count = keep = 1
    if router.get("groups") is not None:
        groups = _map(router, "groups", where + "mlp.router.")
        count, keep = _int(groups, "count", where + "mlp.router.groups."), _int(groups, "keep", where + "mlp.router.groups.")
    if experts % count or keep > count:
        raise ModelConfigError(f"config.json: {where}mlp.router.groups: {count} groups must divide the {experts} experts, and keep "
                               f"{keep} cannot exceed them")
    if top > keep * (experts // count):
        raise ModelConfigError(f"config.json: {where}mlp.router.top {top} exceeds the experts of the {keep} groups that are kept")
    if mlp.get("shared") is not None:
        _int(_map(mlp, "shared", where + "mlp."), "ff", where + "mlp.shared.")


@dataclass(frozen=True)
class MubutarConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embedding_scale: Optional[float]
    logit_scale: Optional[float]
    layers: Tuple[Mapping[str, Any], ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MubutarConfig":
        if not isinstance(d, Mapping):
            raise ModelConfigError("config.json must hold a JSON object")
        arch = d.get("architecture")
        if not isinstance(arch, str):
            archs = d.get("architectures")
            arch = archs[0] if isinstance(archs, (list, tuple)) and archs else None
        if not isinstance(arch, str):
            raise ModelConfigError("config.json lacks required key 'architecture'")
        eps = _num(_map(d, "norm", ""), "eps", "norm.", positive=True)
        emb = None
        if d.get("embedding") is not None and _map(d, "embedding", "").get("scale") is not None:
            emb = _num(d["embedding"], "scale", "embedding.")
        logit = _num(d, "logit_scale", "") if d.get("logit_scale") is not None else None
        entries = d.get("layers")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ModelConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(e, Mapping):
                raise ModelConfigError(f"config.json: {where[:-1]} must be an object")
            _check_mixer(e.get("type"), _map(e, "mixer", where), where + "mixer.", i, [x["mixer"] for x in layers])
            _check_mlp(e.get("mlp"), where)
            layers.append(copy.deepcopy({"type": e["type"], "mixer": dict(e["mixer"]), "mlp": e.get("mlp")}))
        return cls(architecture=arch, vocab_size=_int(d, "vocab", ""), hidden_size=_int(d, "width", ""), norm_eps=eps,
                   embedding_scale=emb, logit_scale=logit, layers=tuple(layers))

    def to_dict(self):
        out = {"architecture": self.architecture, "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps},
               "vocab": self.vocab_size, "width": self.hidden_size}
        if self.embedding_scale is not None:
            out["embedding"] = {"scale": self.embedding_scale}
        if self.logit_scale is not None:
            out["logit_scale"] = self.logit_scale
        return out

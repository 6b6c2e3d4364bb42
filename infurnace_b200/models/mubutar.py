"""Mubutar: the plan builder (configuration -> layers, order, tensor names).

A decoder over a float32 residual stream whose layers have one norm each: h = norm1(x), x += mixer(h) + ff(h), both
sublayers reading the same h.  The embedding's rows and the logits are multiplied by one number each.  The mixer is
grouped-query attention without positions: q, k and v with biases, keys and values of different widths, scores capped
(c * tanh(s / c)), exp(0) beside the keys in the softmax's denominator; a layer may have queries only and read the keys and values of an
earlier layer (its layer call then names that layer's cache entry and stores nothing).  The feed-forward is a gated silu
one, or a mixture of ungated relu² experts: sigmoid scores, chosen by score plus a correction within the best groups of
neighbouring experts (a group counts by its two best), weighted by the chosen scores over their sum, beside a shared expert
of the same form.  A final norm and an untied head follow.  Tensor names: ``embed``, ``l<i>.norm1``,
``l<i>.mix.q|q.b|k|k.b|v|v.b|o``, ``l<i>.mlp.gate|up|down`` (dense), ``l<i>.mlp.router|correction``,
``l<i>.mlp.e<j>.up|down``, ``l<i>.mlp.shared.up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.mubutar import MubutarConfig
from ..config.specs import (
    DenseMLPSpec, EmbeddingSpec, GatedMLPSpec, LayerCall, LMHeadSpec, ModelPlan, ParallelBlockSpec, RMSNormSpec,
    RotaryValueAttentionSpec, RoutedExpertsSpec,
)
from .registry import register_architecture

MAX_POSITIONS = 1 << 20        # positions have no end in this design; block tables need one
DENSE_ACTIVATION = "silu"
EXPERT_ACTIVATION = "relu2"
SINK_SCORE = 0.0               # exp(0) joins the softmax's denominator
GROUP_BEST = 2                 # a group of experts counts by the sum of its two best choice scores
WEIGHT_TERMS = 2               # softmax weights are 32-bit in this design: on tensor cores they enter the sum as two terms


def _mixer(m, p, W, eps):
    own = m.get("kv_from") is None
    return RotaryValueAttentionSpec(
        hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_head_dim=m["vdim"],
        scale=float(m["scale"]), eps=eps, q_proj=p + "q", k_proj=p + "k" if own else None, v_proj=p + "v" if own else None,
        o_proj=p + "o", weight_terms=WEIGHT_TERMS, q_bias=p + "q.b", k_bias=p + "k.b" if own else None,
        v_bias=p + "v.b" if own else None, softcap=float(m["softcap"]) if m.get("softcap") is not None else None,
        sink_score=SINK_SCORE, reads_cache=not own)


def _mlp(mlp, p, W):
    if mlp["kind"] == "dense":
        return GatedMLPSpec(W, mlp["ff"], DENSE_ACTIVATION, p + "gate", p + "up", p + "down")
    router, shared = mlp["router"], mlp.get("shared")
    groups = router.get("groups")
    return RoutedExpertsSpec(
        W, mlp["expert"]["ff"], router["top"], EXPERT_ACTIVATION, p + "router",
        tuple((f"{p}e{j}.up", f"{p}e{j}.down") for j in range(router["experts"])), scoring="sigmoid", correction=p + "correction",
        normalise=True, groups=(int(groups["count"]), int(groups["keep"])) if groups else None, group_best=GROUP_BEST,
        shared=DenseMLPSpec(W, shared["ff"], EXPERT_ACTIVATION, p + "shared.up", p + "shared.down") if shared else None)


def build_mubutar_plan(cfg: MubutarConfig) -> ModelPlan:
    W, eps, V = cfg.hidden_size, cfg.norm_eps, cfg.vocab_size
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        layers.append(ParallelBlockSpec(
            norm=RMSNormSpec(W, eps, p + "norm1"), mixer=_mixer(m, p + "mix.", W, eps),
            ffn=_mlp(layer["mlp"], p + "mlp.", W) if layer["mlp"] is not None else None))
        src = m.get("kv_from")
        schedule.append(LayerCall(i, cache=i) if src is None else LayerCall(i, cache=int(src), store=False))
    return ModelPlan(
        architecture=cfg.architecture, vocab_size=V, hidden_size=W, max_positions=MAX_POSITIONS,
        embedding=EmbeddingSpec(V, W, "embed", scale=1.0 if cfg.embedding_scale is None else cfg.embedding_scale),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=RMSNormSpec(W, eps, "final.norm"),
        lm_head=LMHeadSpec(V, W, "head", tied=False, scale=1.0 if cfg.logit_scale is None else cfg.logit_scale))


register_architecture("Mubutar", MubutarConfig, build_mubutar_plan)

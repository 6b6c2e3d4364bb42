"""Tigelorn: the plan builder (configuration -> layers, order, tensor names).

A pre-norm decoder over a float32 residual stream whose norms store what their factor differs from one by.  The embedding
adds a row of a second table, picked by the token and the one before it.  A layer is x += mixer(norm1(x)), then, where it has
a feed-forward, x += ff(norm2(x)).  Three mixers, in any order given by config.json's ``layers``: ``channel_delta`` (the
gated delta rule with a decay per key channel, behind short convolutions), ``latent_attention`` (queries through a latent of
their own; keys and values from a small cached latent beside one rotated key part shared by the heads, with stretched
rotary frequencies) and ``parallel`` (gated grouped-query attention with unit queries and keys under a sliding window,
beside linear attention with a fixed decay per head; a weighted sum).  The feed-forward is dense with a gelu gate.  A layer may
run with another layer's tensors (``weights_of``): one set of parts, a schedule entry and cache entries of its own.  A final
norm and the embedding table as the head follow.  Tensor names: ``embed``, ``bigram``, ``l<i>.norm1|norm2``,
``l<i>.mix.*`` (``l<i>.mix.left.*`` and ``l<i>.mix.right.*`` in a parallel mixer), ``l<i>.mlp.gate|up|down``, ``final.norm``.
"""
from __future__ import annotations

from ..config.specs import (
    BigramEmbeddingSpec, DeltaRuleSpec, EmbeddingSpec, GatedMLPSpec, LatentAttentionSpec, LayerCall, LMHeadSpec, ModelPlan,
    ParallelMixerSpec, PreNormBlockSpec, RetentionSpec, RMSNormSpec, RotarySpec, RotaryValueAttentionSpec,
)
from ..config.tigelorn import DELTA, LATENT, PARALLEL, TigelornConfig, root_of
from .registry import register_architecture

MAX_POSITIONS = 1 << 20        # positions have no end in this design; block tables need one
ACTIVATION = "gelu_tanh"
NORM_OFFSET = 1.0              # norm weights are stored around zero
UNIT_EPS = 1e-6                # in the length of the delta rule's queries and keys
WEIGHT_TERMS = 2               # softmax weights are 32-bit in this design: on tensor cores they enter the sum as two terms


def _rotary(rot, width, interleaved):
    sc = rot.get("scaling")
    scaling = (float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"])) if sc else None
    return RotarySpec(width, int(rot["dims"]), float(rot["base"]), interleaved=interleaved, scaling=scaling, frequency_dtype="float64")


def _window(m):
    return int(m["mask"]["size"]) if m.get("mask") else None


def _delta(m, p, W, eps):
    return DeltaRuleSpec(
        hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_head_dim=m["vdim"], taps=m["conv"],
        eps=eps, q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", q_conv=p + "q.conv", k_conv=p + "k.conv", v_conv=p + "v.conv",
        beta_proj=p + "b", a_log=p + "A_log", decay_down=p + "a1", decay_up=p + "a2", decay_bias=p + "dt_bias", gate_down=p + "g1",
        gate_up=p + "g2", out_norm=p + "norm", o_proj=p + "o", unit_eps=UNIT_EPS, rank=m.get("rank"))


def _latent(m, p, W, eps):
    rot_dim = int(m.get("rot_dim") or 0)
    return LatentAttentionSpec(
        hidden_size=W, num_heads=m["heads"], head_dim=m["dim"], rot_dim=rot_dim, value_head_dim=m["vdim"], kv_rank=m["kv_rank"],
        scale=float(m["scale"]), eps=eps, q_proj=p + "uq", down_proj=p + "dkv", latent_norm=p + "dkv.norm", k_up=p + "uk", v_up=p + "uv",
        o_proj=p + "o", position=_rotary(m["rot"], rot_dim, True) if rot_dim else None, window=_window(m), q_rank=m["q_rank"],
        q_down=p + "dq", q_norm=p + "dq.norm", weight_terms=WEIGHT_TERMS)


def _parallel(m, p, W, eps):
    left, right = m["left"], m["right"]
    lp, rp = p + "left.", p + "right."
    attention = RotaryValueAttentionSpec(
        hidden_size=W, num_heads=left["heads"], num_kv_heads=left["kv_heads"], head_dim=left["dim"], value_head_dim=left["vdim"],
        scale=float(left["scale"]), eps=eps, q_proj=lp + "q", k_proj=lp + "k", v_proj=lp + "v", o_proj=lp + "o",
        position=_rotary(left["rot"], left["dim"], False) if left.get("rot") else None, window=_window(left), weight_terms=WEIGHT_TERMS,
        q_bias=lp + "q.b", k_bias=lp + "k.b", v_bias=lp + "v.b", unit_qk=True, gate=lp + "g")
    linear = RetentionSpec(
        hidden_size=W, num_heads=right["heads"], head_dim=right["dim"], value_head_dim=right["vdim"],
        decay=tuple(float(x) for x in right["decay"]), key_scale=1.0, eps=eps, q_proj=rp + "q", k_proj=rp + "k", v_proj=rp + "v",
        g_proj=rp + "g", o_proj=rp + "o", input_activation="silu", joint_norm=rp + "norm", gate_activation="sigmoid")
    return ParallelMixerSpec((attention, linear), (float(m["left_scale"]), float(m["right_scale"])))


_MIXERS = {DELTA: _delta, LATENT: _latent, PARALLEL: _parallel}


def build_tigelorn_plan(cfg: TigelornConfig) -> ModelPlan:
    W, eps, V = cfg.hidden_size, cfg.norm_eps, cfg.vocab_size

    def norm(name):
        return RMSNormSpec(W, eps, name, offset=NORM_OFFSET)
    own = [i for i in range(len(cfg.layers)) if root_of(cfg.layers, i) == i]      # layers with tensors
    layers = []
    for i in own:
        layer, p = cfg.layers[i], f"l{i}."
        mlp = layer["mlp"]
        layers.append(PreNormBlockSpec(
            mixer_norm=norm(p + "norm1"), mixer=_MIXERS[layer["type"]](layer["mixer"], p + "mix.", W, eps),
            ffn_norm=norm(p + "norm2") if mlp is not None else None,
            ffn=GatedMLPSpec(W, mlp["ff"], ACTIVATION, p + "mlp.gate", p + "mlp.up", p + "mlp.down") if mlp is not None else None))
    if cfg.bigram is not None:
        embedding = BigramEmbeddingSpec(V, W, "embed", "bigram", cfg.bigram["buckets"], cfg.bigram["mul_prev"], cfg.bigram["mul_cur"])
    else:
        embedding = EmbeddingSpec(V, W, "embed")
    return ModelPlan(
        architecture=cfg.architecture, vocab_size=V, hidden_size=W, max_positions=MAX_POSITIONS, embedding=embedding,
        layers=tuple(layers), schedule=tuple(LayerCall(own.index(root_of(cfg.layers, i)), cache=i) for i in range(len(cfg.layers))),
        final_norm=norm("final.norm"), lm_head=LMHeadSpec(V, W, "embed", tied=True))


register_architecture("Tigelorn", TigelornConfig, build_tigelorn_plan)

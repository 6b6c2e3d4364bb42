"""Grouped-query softmax attention over page streams of keys and values: optional biases, positions on queries, keys and
values, normalised values, queries and keys of unit size, an output gate, a soft cap on the scores, a sink in the softmax, queries over another layer's keys and values."""
from __future__ import annotations

import torch

from ..config.specs import RotaryValueAttentionSpec
from .registry import build_part, fold_residual_norm, register_part, unfolded


class RotaryValueAttention:
    """h -> o_proj(unrotate(attention(q, K, V))).

    q | k | v run as one product (q | k where the description has no value projection: a value head is then its key head
    as projected, before the rotation), the biases added in it.  A part that ``reads_cache`` has the q product alone, which
    then writes the queries in the cache's dtype, and stores nothing.  One kernel rotates the q and k heads on their first rotary_dim entries, divides
    each value head by its root mean square and rotates it over its whole width by the token's position, writes q
    in the cache's dtype and k and v into their page streams (which may differ in width).  The attention kernel reads
    every key and value from the pages, this step's included, keeps scores, softmax weights and sums in float32,
    and rotates each head's summed output back by the query's position before it stores it.  The angles come from
    the rotary parts' per-step tables (cosine and sine of every token's angles, float32).

    With ``unit_qk`` the storing kernel also divides the rotated q and k heads by their root mean square.  With a ``gate``
    its matrix is a further block of rows of the one input product, and one kernel multiplies the heads by the gates'
    sigmoids.  The part can stand inside a :class:`ParallelMixer` whose mixers share their first and last products
    (``w_in``, ``b_in``, ``mix``, ``w_o``)."""

    graph_safe = True

    def __init__(self, spec: RotaryValueAttentionSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.values_are_keys = spec.v_proj is None and not spec.reads_cache
        if self.values_are_keys and (spec.value_head_dim != spec.head_dim or spec.value_norm or spec.value_position is not None):
            raise ValueError("values that are the keys have the keys' width, no norm and no rotation of their own")
        if spec.reads_cache and (spec.value_norm or spec.k_proj is not None or spec.v_proj is not None):
            raise ValueError("a mixer that reads another's keys and values makes none")
        if spec.reads_cache and (spec.unit_qk or spec.gate is not None):
            raise ValueError("queries over another's keys have no norm and no gate")
        pairs = [(p, b) for p, b in ((spec.q_proj, spec.q_bias), (spec.k_proj, spec.k_bias), (spec.v_proj, spec.v_bias)) if p is not None]
        self.qkv_width = sum(weights[p].shape[0] for p, _ in pairs)
        if spec.gate is not None:
            pairs.append((spec.gate, None))
        self.w_in = torch.cat([weights[p] for p, _ in pairs], dim=0).contiguous()
        self.b_in = None
        if any(b is not None for _, b in pairs):          # float32, zeros where a projection has none
            self.b_in = torch.cat([weights[b].float() if b is not None else
                                   torch.zeros(weights[p].shape[0], dtype=torch.float32, device=weights[p].device)
                                   for p, b in pairs], dim=0).contiguous()
        self.w_o = weights[spec.o_proj]
        self.position = build_part(spec.position, weights, runtime) if spec.position is not None else None
        self.value_position = build_part(spec.value_position, weights, runtime) if spec.value_position is not None else None
        if self.value_position is not None and spec.value_position.rotary_dim != spec.value_head_dim:
            raise ValueError("the values are rotated over their whole width")
        import os
        self.exact_weights = os.environ.get("INFURNACE_EXACT_ATTENTION", "0") not in ("", "0")
        self.out_width = spec.num_heads * spec.value_head_dim
        self.joint = not spec.reads_cache                 # may share its products with the mixers beside it
        # what the call of the streams' attention kernel needs beyond the plain softmax
        self.extra = {key: value for key, value in (("softcap", spec.softcap), ("sink", spec.sink_score)) if value is not None}
        if spec.weight_terms != 1:
            self.extra["weight_terms"] = spec.weight_terms
        if spec.unit_qk:                              # |q . k| is at most head_dim
            self.extra["score_bound"] = abs(spec.scale) * spec.head_dim

    can_fold_output = True

    def can_take_folded(self, n):
        can = getattr(self.k, "can_fold_norm", None)
        return bool(can and can(n, self.rt.act_dtype, self.w_in))

    def _plain_on_tensor_cores(self, kv):
        """bfloat16 with keys and values of one width in one tensor: the framework's tensor-core attention kernels run
        (scores and softmax in float32; the weights are rounded to bfloat16 as the left operand of the P V product, which
        accumulates in float32).  Everything else goes to the streams' entry, which takes its tensor-core route where the
        sizes allow (widths of their own for keys and values, a soft cap, a sink) and, when ``exact_weights`` is set, always the
        plain kernel, which keeps the weights in float32 through the sum."""
        s = self.spec
        group = s.num_heads // s.num_kv_heads
        return (not self.exact_weights and s.softcap is None and s.sink_score is None and self.rt.act_dtype == torch.bfloat16 and kv.pages is not None
                and s.head_dim == s.value_head_dim and s.head_dim % 16 == 0 and s.head_dim <= 256 and group <= 16
                and hasattr(self.k, "rotate_rows"))

    def _project(self, h, row_scale, out):
        args = {}
        if row_scale is not None:
            args["row_scale"] = row_scale
        if self.b_in is not None:
            args["bias"] = self.b_in
        self.k.linear(h, self.w_in, out, **args)

    def _queries(self, proj, ctx, call, kv, v_table):
        """The step's queries in the cache's dtype; its keys and values in the pages."""
        s, k = self.spec, self.k
        n = proj.shape[0]
        pk, pv = kv.streams["k"], kv.streams["v"]
        q = ctx.buffer("rva_q", (n, s.num_heads * s.head_dim), self.rt.act_dtype)
        qk_table = self.position.table(ctx) if self.position is not None else None
        extra = {"values_are_keys": True} if self.values_are_keys else {}
        if s.unit_qk:
            extra["qk_eps"] = s.eps
        k.rotary_store(proj[:, :self.qkv_width], s.num_heads, s.num_kv_heads, s.head_dim, s.value_head_dim, qk_table,
                       s.position.rotary_dim if s.position is not None else 0,
                       bool(s.position.interleaved) if s.position is not None else False,
                       s.eps if s.value_norm else None, v_table,
                       bool(s.value_position.interleaved) if s.value_position is not None else False,
                       q, pk, pv, kv.slot_mapping if call.store else None, **extra)
        return q

    def _queries_alone(self, h, row_scale, ctx):
        """The queries of a part that makes no keys: their product writes the cache's dtype."""
        s, k = self.spec, self.k
        q = ctx.buffer("rva_q", (h.shape[0], s.num_heads * s.head_dim), self.rt.act_dtype)
        self._project(h, row_scale, q)
        if self.position is not None:
            k.rotate_rows(q, self.position.table(ctx), s.num_heads, s.head_dim, s.position.rotary_dim, bool(s.position.interleaved))
        return q

    def forward(self, h, ctx, call, fold=None, out=None):
        """``fold``: as :meth:`GatedMLP.forward`'s.  ``out``: where the result goes if it is not folded into the stream (default: a
        buffer of the part's)."""
        s, k = self.spec, self.k
        h, row_scale = unfolded(h)
        n = h.shape[0]
        attn = ctx.buffer("rva_out", (n, self.out_width), self.rt.act_dtype)
        if s.reads_cache:
            self._attend(self._queries_alone(h, row_scale, ctx), attn, ctx, ctx.kv(call.cache),
                         self.value_position.table(ctx) if self.value_position is not None else None)
        else:
            proj = ctx.buffer("rva_proj", (n, self.w_in.shape[0]), torch.float32)
            self._project(h, row_scale, proj)
            self.mix(proj, ctx, call, attn)
        folded = fold_residual_norm(k, ctx, "mixer", attn, self.w_o, fold, self.rt.act_dtype)
        if folded is not None:
            return folded
        delta = out if out is not None else ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(attn, self.w_o, delta)
        return delta

    def mix(self, proj, ctx, call, out, gain=1.0):
        """From the input product's rows (``proj`` [n, rows of w_in], maybe a slice of a wider product) to the rows that the
        output product reads: ``gain`` times the (gated) heads into ``out``, whose rows may be a slice too."""
        s, k = self.spec, self.k
        kv = ctx.kv(call.cache)
        v_table = self.value_position.table(ctx) if self.value_position is not None else None
        q = self._queries(proj, ctx, call, kv, v_table)
        direct = s.gate is None and gain == 1.0 and out.is_contiguous()
        heads = out if direct else ctx.buffer("rva_heads", (proj.shape[0], self.out_width), self.rt.act_dtype)
        self._attend(q, heads, ctx, kv, v_table)
        if not direct:
            k.norm_gate_rows(heads, out, gate=proj[:, self.qkv_width:] if s.gate is not None else None, activation="sigmoid", scale=gain)

    def _attend(self, q, attn, ctx, kv, v_table):
        s, k = self.spec, self.k
        pk, pv = kv.streams["k"], kv.streams["v"]
        if self._plain_on_tensor_cores(kv):
            # the framework's tensor-core attention over the entry's one tensor of keys and values, then the turn back
            k.paged_attention(q, s.num_heads, s.num_kv_heads, s.head_dim, kv.pages, kv.block_tables, ctx.cu_q, ctx.seq_lens, attn,
                              s.scale, s.window or 0, ctx.max_q_len, ctx.max_seq_len, min_q_len=ctx.min_q_len,
                              **{key: self.extra[key] for key in ("weight_terms", "score_bound") if key in self.extra})
            if v_table is not None:
                k.rotate_rows(attn, v_table, s.num_heads, s.value_head_dim, s.value_head_dim, bool(s.value_position.interleaved),
                              back=True)
        else:
            k.paged_attention_streams(q, s.num_heads, s.num_kv_heads, s.head_dim, s.value_head_dim, pk, pv, kv.block_tables,
                                      ctx.cu_q, ctx.seq_lens, attn, s.scale, s.window or 0, v_table,
                                      bool(s.value_position.interleaved) if s.value_position is not None else False,
                                      max_q_len=ctx.max_q_len, max_seq_len=ctx.max_seq_len, min_q_len=ctx.min_q_len,
                                      exact=self.exact_weights, **self.extra)


register_part(RotaryValueAttentionSpec, RotaryValueAttention)

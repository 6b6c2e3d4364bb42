"""Recurrent mixers whose state lives in the request's state slot: the HGRN2 gated recurrence, retention with a fixed
decay per head, RWKV-style time mixing, the gated delta rule (all four a matrix state per head), the element-wise minGRU and the real-gated
linear recurrent unit behind a short convolution."""
from __future__ import annotations

import torch

from ..config.specs import DeltaRuleSpec, GatedRecurrenceSpec, GatedUnitSpec, RealGatedRecurrenceSpec, RetentionSpec, TimeMixSpec
from ..errors import WeightError
from .registry import fold_residual_norm, register_part, unfolded


class GatedRecurrence:
    """h -> o_proj(norm(S^T q)) with S <- diag(f) S + (1 - f) v^T per head.

    The three projections run as one product against their row-wise concatenation (exact) into float32, because
    everything that enters the recurrence is 32-bit.  One kernel then applies silu to q and the gate formula to f,
    walks this step's tokens of every request in order from the state its slot holds (zero when the slot was
    granted), writes the state back and normalises each head's output.  A whole prompt, a portion and a single
    decoded token are the same call: the state carries what came before."""

    graph_safe = True     # launches depend on the step's sizes only

    def __init__(self, spec: GatedRecurrenceSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.w_qfv = torch.cat((weights[spec.q_proj], weights[spec.f_proj], weights[spec.v_proj]), dim=0).contiguous()
        self.w_o = weights[spec.o_proj]
        self.bias, self.lower, self.norm_w = weights[spec.f_bias], weights[spec.lower], weights[spec.out_norm]
        self.hd = spec.num_heads * spec.head_dim
        self.hv = spec.num_heads * spec.value_head_dim
        slabs = getattr(self.k, "gated_scan_slabs", None)
        self.slabs = slabs(spec.head_dim, spec.value_head_dim) if slabs else 1

    def forward(self, h, ctx, call):
        s, k = self.spec, self.k
        n = h.shape[0]
        proj = ctx.buffer("gr_proj", (n, 2 * self.hd + self.hv), torch.float32)
        k.linear(h, self.w_qfv, proj)
        out = ctx.buffer("gr_out", (n, self.hv), self.rt.act_dtype)
        raw = ctx.buffer("gr_raw", (n, self.hv), torch.float32) if self.slabs > 1 else None
        k.gated_scan(proj, 0, self.hd, 2 * self.hd, self.bias, self.lower, self.norm_w, s.eps, ctx.state(call.cache),
                     ctx.state_slots, ctx.cu_q, ctx.seq_lens, out, s.num_heads, s.head_dim, s.value_head_dim, raw=raw,
                     max_q_len=ctx.max_q_len)
        delta = ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta


register_part(GatedRecurrenceSpec, GatedRecurrence)


class Retention:
    """h -> o_proj(norm(S^T q) * act(G h)) with S <- decay_h S + (k * key_scale) v^T per head.

    q | k | v | g run as one product into float32 (what enters the recurrence is 32-bit).  The recurrence kernel is
    the framework's walk of a matrix state per head (``linear_scan``) with a constant decay per head; it divides each
    head's output by its root mean square and multiplies by silu of the gate columns before it writes the rows that
    ``o_proj`` reads.  Where the heads are normed together, or the gate is a sigmoid, the recurrence leaves its float32
    outputs and a second kernel does both.  q, k and v may pass silu as the recurrence reads them.  A prompt, a portion and a
    decoded token are the same call: the slot's state carries the past.  The part can share its first and last products with
    mixers beside it (``w_in``, ``mix``, ``w_o``)."""

    graph_safe = True
    can_fold_output = True
    joint = True
    b_in = None

    def can_take_folded(self, n):
        can = getattr(self.k, "can_fold_norm", None)
        return bool(can and can(n, self.rt.act_dtype, self.w_in))

    def __init__(self, spec: RetentionSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        if spec.input_activation not in (None, "silu") or spec.gate_activation not in ("silu", "sigmoid"):
            raise ValueError("retention: the inputs' activation is silu or none, the gate's silu or sigmoid")
        self.w_in = torch.cat([weights[n] for n in (spec.q_proj, spec.k_proj, spec.v_proj, spec.g_proj)], dim=0).contiguous()
        self.w_o = weights[spec.o_proj]
        self.joint_w = weights[spec.joint_norm].float().contiguous() if spec.joint_norm is not None else None
        self.decay = torch.tensor(spec.decay, dtype=torch.float32, device=runtime.device)
        self.hd = spec.num_heads * spec.head_dim
        self.hv = self.out_width = spec.num_heads * spec.value_head_dim

    def forward(self, h, ctx, call, fold=None):
        s, k = self.spec, self.k
        h, row_scale = unfolded(h)
        n = h.shape[0]
        proj = ctx.buffer("ret_proj", (n, self.w_in.shape[0]), torch.float32)
        k.linear(h, self.w_in, proj, **({"row_scale": row_scale} if row_scale is not None else {}))
        out = ctx.buffer("ret_out", (n, self.hv), self.rt.act_dtype)
        self.mix(proj, ctx, call, out)
        folded = fold_residual_norm(k, ctx, "mixer", out, self.w_o, fold, self.rt.act_dtype)
        if folded is not None:
            return folded
        delta = ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta

    def mix(self, proj, ctx, call, out, gain=1.0):
        """From the input product's rows (``proj``, maybe a slice of a wider product) to ``gain`` times the gated heads in
        ``out``, whose rows may be a slice too."""
        s, k, hd, hv = self.spec, self.k, self.hd, self.hv
        n = proj.shape[0]
        one_pass = self.joint_w is None and s.gate_activation == "silu" and gain == 1.0 and out.is_contiguous()
        gate = proj[:, 2 * hd + hv:]
        extra = {"activation": s.input_activation} if s.input_activation is not None else {}
        o = out if one_pass else ctx.buffer("ret_raw", (n, hv), torch.float32)
        k.linear_scan(proj[:, :hd], proj[:, hd:2 * hd], proj[:, 2 * hd:2 * hd + hv], None, s.num_heads, s.head_dim,
                      s.value_head_dim, ctx.state(call.cache), ctx.state_slots, ctx.cu_q, ctx.seq_lens, o, s.eps,
                      decay=self.decay, key_scale=s.key_scale, max_q_len=ctx.max_q_len,
                      **({"gate": gate} if one_pass else {"finish": False}), **extra)
        if not one_pass:
            k.norm_gate_rows(o, out, groups=1 if self.joint_w is not None else s.num_heads, weight=self.joint_w, eps=s.eps,
                             gate=gate, activation=s.gate_activation, scale=gain)


register_part(RetentionSpec, Retention)


class TimeMix:
    """RWKV-style time mixing over two cache entries: the matrix state per head, and the previous token's input.

    One kernel forms the five blends of each token with the one before it (the slot's saved row for the first token
    of a step) and saves the step's last row.  r, k, v, g and the decay's bottleneck read their blends through the
    framework's products (into float32; the bottleneck's tanh is its product's epilogue); the recurrence kernel
    turns the raw decay into exp(-exp(. + w0)), reads each output from the state BEFORE the token's update with the
    bonus on the token's own k v^T, and finishes with the per-head unit norm, the stored norm weight and the gate."""

    graph_safe = True

    def __init__(self, spec: TimeMixSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.mu = torch.stack([weights[n].to(torch.float32) for n in spec.mu], dim=0).contiguous()
        self.w_r, self.w_k, self.w_v, self.w_g = (weights[n] for n in (spec.r_proj, spec.k_proj, spec.v_proj, spec.g_proj))
        self.w1, self.w2, self.w0 = weights[spec.w1], weights[spec.w2], weights[spec.w0]
        self.rank = self.w1.shape[0]
        self.bonus = weights[spec.bonus].reshape(-1).contiguous()
        self.norm_w = weights[spec.out_norm]
        self.w_o = weights[spec.o_proj]
        self.hd = spec.num_heads * spec.head_dim

    def forward(self, h, ctx, call):
        s, k, hd = self.spec, self.k, self.hd
        n, W = h.shape
        mixes = ctx.buffer("tm_mixes", (5 * n, W), self.rt.act_dtype).view(5, n, W)
        k.token_shift_mix(h, ctx.state((call.cache, 1)), ctx.state_slots, ctx.cu_q, ctx.seq_lens, self.mu, mixes)
        proj = [ctx.buffer("tm_" + name, (n, hd), torch.float32) for name in ("r", "k", "v", "g", "w")]
        for j, w in enumerate((self.w_r, self.w_k, self.w_v, self.w_g)):
            k.linear(mixes[j], w, proj[j])
        low = ctx.buffer("tm_low", (n, self.rank), self.rt.act_dtype)
        k.linear(mixes[4], self.w1, low, epilogue="tanh")
        k.linear(low, self.w2, proj[4])
        out = ctx.buffer("tm_out", (n, hd), self.rt.act_dtype)
        k.linear_scan(proj[0], proj[1], proj[2], proj[4], s.num_heads, s.head_dim, s.head_dim, ctx.state((call.cache, 0)),
                      ctx.state_slots, ctx.cu_q, ctx.seq_lens, out, s.eps, w_bias=self.w0, bonus=self.bonus,
                      norm_weight=self.norm_w, gate=proj[3], max_q_len=ctx.max_q_len)
        delta = ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta


register_part(TimeMixSpec, TimeMix)


class DeltaRule:
    """h -> o_proj(norm(S^T q) * sigmoid(g2 g1 h)); S <- diag(g) S, S <- S + k (beta (v - S^T k))^T per head.

    q | k | v | beta | the two bottlenecks run as one product into float32.  One kernel runs the short convolutions over each
    request's tokens from the inputs its slot kept (cache entry 1), applies silu and makes q and k unit vectors, forms beta,
    and hands the bottlenecks on in the products' dtype.  Their two second matrices are one product against a
    block-diagonal matrix (exact: the other block is zeros) into float32.  The recurrence kernel forms the decays in float32
    from those rows and walks each request's tokens from the slot's state (cache entry 0), or, for long portions, runs chunks
    of 16 tokens side by side as far as they do not depend on the state; each head's norm and gate follow."""

    graph_safe = True
    can_fold_output = True

    def __init__(self, spec: DeltaRuleSpec, weights, runtime):
        self.spec = s = spec
        self.rt = runtime
        self.k = runtime.kernels
        H, D, V = s.num_heads, s.head_dim, s.value_head_dim
        if H % s.num_kv_heads:
            raise ValueError("delta rule: the heads are a multiple of the query/key heads")
        down = [weights[n] for n in (s.decay_down, s.gate_down)]
        up = [weights[n] for n in (s.decay_up, s.gate_up)]
        if any(d.shape[0] != u.shape[1] for d, u in zip(down, up)):
            raise WeightError(f"weights do not match the model: {s.decay_up} / {s.gate_up} do not take what {s.decay_down} / "
                              f"{s.gate_down} give")
        self.w_in = torch.cat([weights[n] for n in (s.q_proj, s.k_proj, s.v_proj, s.beta_proj)] + down, dim=0).contiguous()
        self.low_width = sum(d.shape[0] for d in down)
        self.low_cols = -(-self.low_width // 8) * 8       # the second product's k: a multiple of 8, zeros beyond
        w_up = torch.zeros((H * (D + V), self.low_cols), dtype=up[0].dtype, device=up[0].device)
        w_up[:H * D, :down[0].shape[0]] = up[0]
        w_up[H * D:, down[0].shape[0]:self.low_width] = up[1]
        self.w_up = w_up
        f32 = lambda t: t.to(torch.float32).contiguous()      # small parameters: the kernels read float32
        self.taps = f32(torch.cat([weights[n] for n in (s.q_conv, s.k_conv, s.v_conv)], dim=0))
        self.rate = torch.exp(f32(weights[s.a_log]))
        self.decay_bias, self.norm_w = f32(weights[s.decay_bias]), f32(weights[s.out_norm])
        self.w_o = weights[s.o_proj]

    def can_take_folded(self, n):
        can = getattr(self.k, "can_fold_norm", None)
        return bool(can and can(n, self.rt.act_dtype, self.w_in))

    def forward(self, h, ctx, call, fold=None):
        s, k = self.spec, self.k
        h, row_scale = unfolded(h)
        n = h.shape[0]
        H, G, D, V = s.num_heads, s.num_kv_heads, s.head_dim, s.value_head_dim
        proj = ctx.buffer("dr_proj", (n, self.w_in.shape[0]), torch.float32)
        k.linear(h, self.w_in, proj, **({"row_scale": row_scale} if row_scale is not None else {}))
        qkv = ctx.buffer("dr_qkv", (n, s.channels), torch.float32)
        beta = ctx.buffer("dr_beta", (n, H), torch.float32)
        low = ctx.buffer("dr_low", (n, self.low_cols), self.rt.act_dtype)
        k.delta_prepare(proj, G, H, D, V, self.taps, s.unit_eps, ctx.state((call.cache, 1)), ctx.state_slots, ctx.cu_q, ctx.seq_lens,
                        ctx.req_index, qkv, beta, low, self.low_width)
        up = ctx.buffer("dr_up", (n, H * (D + V)), torch.float32)
        k.linear(low, self.w_up, up)
        out = ctx.buffer("dr_out", (n, H * V), self.rt.act_dtype)
        k.delta_rule(qkv, up, beta, G, H, D, V, self.rate, self.decay_bias, self.norm_w, s.eps, ctx.state((call.cache, 0)),
                     ctx.state_slots, ctx.cu_q, ctx.seq_lens, out, max_q_len=ctx.max_q_len)
        folded = fold_residual_norm(k, ctx, "mixer", out, self.w_o, fold, self.rt.act_dtype)
        if folded is not None:
            return folded
        delta = ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta


register_part(DeltaRuleSpec, DeltaRule)


class GatedUnit:
    """minGRU: z | x | g run as one product into float32; one kernel adds the biases, forms gate and candidate,
    walks each request's tokens element by element from the slot's state and writes S * silu(g)."""

    graph_safe = True
    delta_buffer = "delta_unit"

    def __init__(self, spec: GatedUnitSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.w_all = torch.cat([weights[n] for n in (spec.z_proj, spec.x_proj, spec.g_proj)], dim=0).contiguous()
        self.z_bias, self.x_bias = weights[spec.z_bias], weights[spec.x_bias]
        self.w_o = weights[spec.o_proj]

    def forward(self, h, ctx, call):
        s, k = self.spec, self.k
        n = h.shape[0]
        proj = ctx.buffer("gu_proj", (n, 3 * s.width), torch.float32)
        k.linear(h, self.w_all, proj)
        out = ctx.buffer("gu_out", (n, s.width), self.rt.act_dtype)
        k.gated_unit_scan(proj, self.z_bias, self.x_bias, ctx.state(call.cache), ctx.state_slots, ctx.cu_q, ctx.seq_lens, out,
                          max_q_len=ctx.max_q_len)
        delta = ctx.buffer("delta_unit", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta


register_part(GatedUnitSpec, GatedUnit)


class RealGatedRecurrence:
    """h -> o_proj(S * gelu_tanh(Y h + by)), S <- a S + sqrt(1 - a^2) * i * u per channel, u = conv(X h + bx).

    y | x run as one product into float32.  One kernel adds the x bias, runs the short causal convolution over each
    request's tokens from the inputs its slot kept (cache entry 1) and writes u twice: float32 for the recurrence and, in the
    products' dtype, block by block for the gates.  The two block-diagonal gate matrices are one grouped product (the
    framework's grouped product with a block in an expert's place: r | i of a block are the rows of one matrix) into
    float32 (where the operands are bfloat16 and the description asks for two terms, u enters as its rounding and what the
    rounding left out against the matrix repeated along k).  The recurrence kernel adds the gates' biases, forms sigmoid, softplus, the decay and the input term in float32,
    walks each request's tokens from the slot's state (cache entry 0; long portions in chunks side by side) and multiplies
    by the gelu branch.  A prompt, a portion and a decoded token are the same calls: the slot carries the past."""

    graph_safe = True

    def __init__(self, spec: RealGatedRecurrenceSpec, weights, runtime):
        self.spec = s = spec
        self.rt = runtime
        self.k = runtime.kernels
        f32 = lambda name: weights[name].to(torch.float32).contiguous()      # small vectors: the kernels read float32
        self.w_yx = torch.cat((weights[s.y_proj], weights[s.x_proj]), dim=0).contiguous()
        self.y_bias, self.x_bias = f32(s.y_bias), f32(s.x_bias)
        self.conv_w, self.conv_b = f32(s.conv), f32(s.conv_bias)
        self.w_gates = torch.cat((weights[s.a_gate], weights[s.x_gate]), dim=1).contiguous()      # [blocks, 2 bs, bs]
        # two terms of u (bfloat16 operands only): the matrix repeated along k meets [roundings | what they left out]
        self.terms = 2 if s.gate_terms == 2 and runtime.act_dtype == torch.bfloat16 else 1
        if self.terms == 2:
            self.w_gates = torch.cat((self.w_gates, self.w_gates), dim=2).contiguous()           # [blocks, 2 bs, 2 bs]
        self.a_bias, self.i_bias = f32(s.a_bias).reshape(-1), f32(s.x_bias_gate).reshape(-1)
        self.decay = f32(s.decay)
        self.w_o = weights[s.o_proj]

    def _segment(self, n):
        """Rows of a block's segment in the grouped product, and the tile of the tcgen05 route (0: the other route)."""
        k = self.k
        ok = getattr(k, "moe_grouped_tc_ok", None)
        if ok is not None and ok(n * self.spec.blocks, self.rt.act_dtype, self.w_gates):
            t = k.MOE_TILE
            return -(-n // t) * t, t
        return n, 0

    def forward(self, h, ctx, call):
        s, k = self.spec, self.k
        n = h.shape[0]
        W, B = s.width, s.blocks
        bs = W // B
        act = self.rt.act_dtype
        proj = ctx.buffer("rg_proj", (n, 2 * W), torch.float32)
        k.linear(h, self.w_yx, proj)
        seg, tile = self._segment(n)
        cap, _ = self._segment(ctx.max_rows)
        u = ctx.buffer("rg_u", (n, W), torch.float32)
        kb = self.terms * bs
        ub = ctx.buffer("rg_u_blocks", (B * seg, kb), act, rows=B * cap).view(B, seg, kb)
        offsets = ctx.buffer("rg_offsets", (B + 1,), torch.int32, rows=B + 1)
        tiles = ctx.buffer("rg_tiles", (B * seg // tile,), torch.int32, rows=B * cap // tile) if tile else None
        k.rglru_conv(proj, W, self.x_bias, self.conv_w, self.conv_b, ctx.state((call.cache, 1)), ctx.state_slots, ctx.cu_q,
                     ctx.seq_lens, ctx.req_index, u, ub, offsets, tiles, tile)
        gates = ctx.buffer("rg_gates", (B * seg, 2 * bs), torch.float32, rows=B * cap)
        if tile:
            k.moe_linear_grouped(ub.view(B * seg, kb), self.w_gates, tiles, gates)
        else:
            k.moe_linear(ub.view(B * seg, kb), self.w_gates, offsets, None, 1, gates)
        out = ctx.buffer("rg_out", (n, W), act)
        k.rglru_scan(gates.view(B, seg, 2 * bs), self.a_bias, self.i_bias, self.decay, s.decay_scale, u, proj, 0, self.y_bias,
                     ctx.state((call.cache, 0)), ctx.state_slots, ctx.cu_q, ctx.seq_lens, out, max_q_len=ctx.max_q_len)
        delta = ctx.buffer("delta_mixer", (n, s.hidden_size), torch.float32)
        k.linear(out, self.w_o, delta)
        return delta


register_part(RealGatedRecurrenceSpec, RealGatedRecurrence)

"""Several mixers side by side on one input."""
from __future__ import annotations

import torch

from ..config.specs import LayerCall, ParallelMixerSpec
from .registry import build_part, fold_residual_norm, register_part, unfolded


class WeightedSum:
    """The results of mixers that ran side by side, not yet added up: ``terms`` = [(float32 tensor, scale), ...].  A
    block whose stream update can form the sum in its own pass asks for this (``weighted=True``)."""
    __slots__ = ("terms",)

    def __init__(self, terms):
        self.terms = terms


class ParallelMixer:
    """h -> sum_i scales[i] * mixers[i](h).  Mixer i keeps cache entry ``(call.cache, i)``.

    Mixers that all offer it (``joint``) share their products: one against their input matrices one below the other, whose
    slices they read, and one against their output matrices side by side, over rows in which mixer i has put scales[i] times
    what its own output product would read.  The sum then happens inside that product.  Else the weighted sum is one
    small kernel per mixer over their float32 results, or the caller takes a :class:`WeightedSum` of two whose results lie
    in buffers of their own."""

    def __init__(self, spec: ParallelMixerSpec, weights, runtime):
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.mixers = [build_part(m, weights, runtime) for m in spec.mixers]
        self.joint = all(getattr(m, "joint", False) for m in self.mixers)
        names = [getattr(m, "delta_buffer", "delta_mixer") for m in self.mixers]
        self.can_return_weighted = not self.joint and len(set(names)) == len(names)
        self.can_fold_output = self.joint
        if self.joint:
            self.w_in = torch.cat([m.w_in for m in self.mixers], dim=0).contiguous()
            self.w_o = torch.cat([m.w_o for m in self.mixers], dim=1).contiguous()
            self.b_in = None
            if any(m.b_in is not None for m in self.mixers):
                self.b_in = torch.cat([m.b_in if m.b_in is not None else
                                       torch.zeros(m.w_in.shape[0], dtype=torch.float32, device=m.w_in.device)
                                       for m in self.mixers]).contiguous()
            self.in_widths = [m.w_in.shape[0] for m in self.mixers]
            for m in self.mixers:                     # the parts' own copies have no reader
                m.w_in = m.b_in = m.w_o = None

    def can_take_folded(self, n):
        can = getattr(self.k, "can_fold_norm", None)
        return bool(self.joint and can and can(n, self.rt.act_dtype, self.w_in))

    @property
    def graph_safe(self):
        return all(getattr(m, "graph_safe", False) for m in self.mixers)

    def _joint_forward(self, h, ctx, call, fold):
        k = self.k
        h, row_scale = unfolded(h)
        n = h.shape[0]
        proj = ctx.buffer("pm_proj", (n, self.w_in.shape[0]), torch.float32)
        args = {} if row_scale is None else {"row_scale": row_scale}
        if self.b_in is not None:
            args["bias"] = self.b_in
        k.linear(h, self.w_in, proj, **args)
        rows = ctx.buffer("pm_rows", (n, self.w_o.shape[1]), self.rt.act_dtype)
        at = col = 0
        for i, (mixer, scale, width) in enumerate(zip(self.mixers, self.spec.scales, self.in_widths)):
            mixer.mix(proj[:, at:at + width], ctx, LayerCall(call.layer, (call.cache, i), call.store),
                      rows[:, col:col + mixer.out_width], gain=scale)
            at, col = at + width, col + mixer.out_width
        folded = fold_residual_norm(k, ctx, "mixer", rows, self.w_o, fold, self.rt.act_dtype)
        if folded is not None:
            return folded
        delta = ctx.buffer("delta_mixer", (n, self.w_o.shape[0]), torch.float32)
        k.linear(rows, self.w_o, delta)
        return delta

    def forward(self, h, ctx, call, weighted=False, fold=None):
        if self.joint:
            return self._joint_forward(h, ctx, call, fold)
        calls = [LayerCall(call.layer, (call.cache, i), call.store) for i in range(len(self.mixers))]
        if weighted and len(self.mixers) == 2 and self.can_return_weighted:
            return WeightedSum([(m.forward(h, ctx, c), scale) for m, c, scale in zip(self.mixers, calls, self.spec.scales)])
        total = None
        for m, c, scale in zip(self.mixers, calls, self.spec.scales):      # a result is added before the next mixer writes its own
            d = m.forward(h, ctx, c)
            if total is None:
                total = ctx.buffer("delta_parallel", d.shape, torch.float32)
                self.k.scaled_sum(total, d, scale, accumulate=False)
            else:
                self.k.scaled_sum(total, d, scale, accumulate=True)
        return total


register_part(ParallelMixerSpec, ParallelMixer)

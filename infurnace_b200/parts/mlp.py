"""The dense gated feed-forward."""
from __future__ import annotations

import torch

from ..config.specs import DenseMLPSpec, GatedMLPSpec
from ..errors import ModelConfigError
from .registry import fold_residual_norm, register_part, unfolded


class GatedMLP:
    """down(act(gate(h)) * up(h)), act silu or the tanh form of gelu (src/infurnace/executor/tinygrad/model.py:146-148).
    gate and up run as one product against their row-wise concatenation (exact), with the
    activation and the product of the two halves in that kernel's epilogue."""

    graph_safe = True     # launches depend on the step's sizes only, never on values read on the host
    EPILOGUES = {"silu": "silu_gate", "gelu_tanh": "gelu_gate"}

    def __init__(self, spec: GatedMLPSpec, weights, runtime):
        if spec.activation not in self.EPILOGUES:
            raise ModelConfigError(f"activation {spec.activation!r}: the gated feed-forward has {', '.join(self.EPILOGUES)}")
        self.epilogue = self.EPILOGUES[spec.activation]
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.w_gate_up = torch.cat((weights[spec.gate_proj], weights[spec.up_proj]), dim=0).contiguous()
        self.w_down = weights[spec.down_proj]

    can_fold_output = True

    def can_take_folded(self, n):
        can = getattr(self.k, "can_fold_norm", None)
        return bool(can and can(n, self.rt.act_dtype, self.w_gate_up, "silu_gate"))

    def forward(self, h, ctx, fold=None, out=None):
        """``out``: where the result goes if it is not folded into the stream (default: a buffer of the part's)."""
        h, row_scale = unfolded(h)
        n = h.shape[0]
        act = ctx.buffer("ffn_act", (n, self.spec.intermediate_size), self.rt.act_dtype)
        if row_scale is not None:
            self.k.linear(h, self.w_gate_up, act, epilogue=self.epilogue, row_scale=row_scale)
        else:
            self.k.linear(h, self.w_gate_up, act, epilogue=self.epilogue)
        folded = fold_residual_norm(self.k, ctx, "ffn", act, self.w_down, fold, self.rt.act_dtype)
        if folded is not None:
            return folded
        delta = out if out is not None else ctx.buffer("delta_ffn", (n, self.spec.hidden_size), torch.float32)
        self.k.linear(act, self.w_down, delta)
        return delta


register_part(GatedMLPSpec, GatedMLP)


class DenseMLP:
    """down(act(up(h))) with the activation in the epilogue of the first product; the result is float32."""

    graph_safe = True
    ACTIVATIONS = ("relu2", "silu", "gelu_tanh")

    def __init__(self, spec: DenseMLPSpec, weights, runtime):
        if spec.activation not in self.ACTIVATIONS:
            raise ModelConfigError(f"activation {spec.activation!r}: the dense feed-forward has {', '.join(self.ACTIVATIONS)}")
        self.spec = spec
        self.rt = runtime
        self.k = runtime.kernels
        self.w_up = weights[spec.up_proj]
        self.w_down = weights[spec.down_proj]

    def forward(self, h, ctx, fold=None, out=None):
        n = h.shape[0]
        act = ctx.buffer("ffn_act", (n, self.spec.intermediate_size), self.rt.act_dtype)
        self.k.linear(h, self.w_up, act, epilogue=self.spec.activation)
        delta = out if out is not None else ctx.buffer("delta_ffn", (n, self.spec.hidden_size), torch.float32)
        self.k.linear(act, self.w_down, delta)
        return delta


register_part(DenseMLPSpec, DenseMLP)

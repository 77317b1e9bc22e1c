"""Gated feed-forward: down(act(gate(x)) * up(x)), act = SiLU (src/qwen.rs:57-68,
silu(a) = a / (1 + exp(-a)) src/kernels.rs:1416-1426) or, with ``activation: gelu_tanh``,
0.5 a (1 + tanh(sqrt(2/pi) (a + 0.044715 a^3))).  The gate and up matrices are stacked at
load into one [2I, H] matrix so one product reads the input once.

``plain_mlp``: the form without a gate, down(act(up(x))), act one of kernels.PLAIN_ACTS (the exact GELU
or the square of relu), applied in the up product's epilogue."""
from __future__ import annotations

import torch

from .. import kernels
from .base import Part, TensorWant, register_part
from .linear import Linear


class GatedMLP(Part):
    category = "ffn"

    def __init__(self, spec, compute):
        super().__init__(spec, compute)
        self.hidden_size = int(spec.params["hidden_size"])
        self.intermediate_size = int(spec.params["intermediate_size"])
        self.activation = act = spec.params.get("activation", "silu")
        if act not in kernels.GATED_ACTS:
            raise ValueError(f"gated_mlp: activation {act!r} has no kernel (known: {', '.join(kernels.GATED_ACTS)})")
        self.gate_up = self.down = None

    def wants(self):
        h, i = self.hidden_size, self.intermediate_size
        return {"gate": TensorWant((i, h)), "up": TensorWant((i, h)), "down": TensorWant((h, i))}

    def load(self, tensors):
        self.gate_up = Linear(torch.cat([tensors["gate"], tensors["up"]], dim=0))
        self.down = Linear(tensors["down"])

    def kernel_units(self):
        if self.activation == "silu":
            return kernels.gemm_units(self.compute) + [("elementwise", ())]
        return kernels.gated_units(self.compute, self.activation)

    #: forward takes ``then_norm`` and may be given kernels.UnscaledRows for ``h``
    links_norms = True

    def set_output_scale(self, scale):
        """``scale`` (float32 [hidden]) multiplies what the feed-forward adds."""
        self.down.out_scale = scale

    def forward(self, ctx, h, residual, then_norm=None):
        """``h``: the normed activations, or kernels.UnscaledRows.  ``then_norm``: the RMSNorm that
        reads the residual next; returns that norm's input where the down product could leave it."""
        rows = h.rows if isinstance(h, kernels.UnscaledRows) else h
        a = torch.empty((rows.shape[0], self.intermediate_size), dtype=rows.dtype, device=rows.device)
        kernels.gemm_gated(h, self.gate_up.weight, a, self.activation)
        return self.down.add_into(a, residual, then_norm)

    def weight_bytes(self):
        return self.gate_up.bytes() + self.down.bytes()


class PlainMLP(Part):
    category = "ffn"
    links_norms = True

    def __init__(self, spec, compute):
        super().__init__(spec, compute)
        self.hidden_size = int(spec.params["hidden_size"])
        self.intermediate_size = int(spec.params["intermediate_size"])
        self.activation = act = spec.params.get("activation", "gelu")
        if act not in kernels.PLAIN_ACTS or act is None:
            raise ValueError(f"plain_mlp: activation {act!r} has no kernel "
                             f"(known: {', '.join(a for a in kernels.PLAIN_ACTS if a)})")
        self.up = self.down = None

    def wants(self):
        h, i = self.hidden_size, self.intermediate_size
        return {"up": TensorWant((i, h)), "down": TensorWant((h, i))}

    def load(self, tensors):
        self.up, self.down = Linear(tensors["up"]), Linear(tensors["down"])

    def set_output_scale(self, scale):
        self.down.out_scale = scale

    def kernel_units(self):
        return kernels.gemm_units(self.compute)

    def forward(self, ctx, h, residual, then_norm=None):
        return self.down.add_into(self.up(h, act=self.activation), residual, then_norm)

    def weight_bytes(self):
        return self.up.bytes() + self.down.bytes()


register_part("ffn", "gated_mlp", GatedMLP)
register_part("ffn", "plain_mlp", PlainMLP)

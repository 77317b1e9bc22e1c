"""Matrix memory with exponential gates (the mLSTM of the xLSTM family): a recurrent mixer whose state
per head is a matrix S [dim, vdim], a vector n [dim] and a running maximum m.

For one token, with h the mixer's input:
  q = W_q h * dim^-1/2, k = W_k h (heads x dim), v = W_v h (heads x vdim);
  i = cap tanh((W_i h + b_i) / cap),  f = logsigmoid(cap tanh((W_f h + b_f) / cap)), one each per head;
  m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n <- the same with k alone;
  o = S^T q / (max(|n . q|, e^(-m')) + 1e-6)      (S, n and m start at zero);
  each head's o divided by its root mean square (eps), the heads side by side times ``norm``, times
  sigmoid(W_g h), then W_o, added into the residual.

The five projections that enter the recurrence and the gate's are one product written in float32,
[q | k | v | g | i | f]; gates, exponentials, the state, the read-out and the norm are float32 work.
Per sequence the part keeps S, and n with m.  Parameters: hidden_size, heads, dim, vdim, gate_cap,
norm_eps, out_scale.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.pool import StateNeed
from .base import Part, TensorWant, register_part
from .linear import Linear


class MatrixMemory(Part):
    category = "mixer"

    def __init__(self, spec, compute):
        super().__init__(spec, compute)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.heads, self.dim, self.vdim = int(p["heads"]), int(p["dim"]), int(p["vdim"])
        self.cap = float(p.get("gate_cap") or 0.0)
        self.eps = float(p["norm_eps"])
        self.out_scale = float(p.get("out_scale", 1.0))
        if self.heads < 1 or self.vdim < 1:
            raise ValueError("matrix_memory: needs at least one head and a value size of at least 1")
        if not 1 <= self.dim <= 256:
            raise ValueError(f"matrix_memory: heads of {self.dim} are not supported by the kernel (1 to 256)")
        if self.cap < 0:
            raise ValueError(f"matrix_memory: gate_cap must not be negative, got {self.cap}")
        self.hd, self.hv = self.heads * self.dim, self.heads * self.vdim
        self.proj = self.o = self.norm = None

    def wants(self):
        h, n = self.hidden_size, self.heads
        return {"q": TensorWant((self.hd, h)), "k": TensorWant((self.hd, h)), "v": TensorWant((self.hv, h)),
                "g": TensorWant((self.hv, h)), "i": TensorWant((n, h)), "f": TensorWant((n, h)),
                "i_bias": TensorWant((n,), "vector"), "f_bias": TensorWant((n,), "vector"),
                "norm": TensorWant((self.hv,), "vector"), "o": TensorWant((h, self.hv))}

    def load(self, t):
        zeros = torch.zeros(2 * (self.hd + self.hv), dtype=torch.float32, device=t["i_bias"].device)
        bias = torch.cat([zeros, t["i_bias"].to(torch.float32), t["f_bias"].to(torch.float32)])
        self.proj = Linear.stacked([t[n] for n in ("q", "k", "v", "g", "i", "f")], bias, multiple=4)
        self.o, self.norm = Linear(t["o"]), t["norm"].to(torch.float32).contiguous()

    #: forward takes ``then_norm`` and may be given kernels.UnscaledRows for ``h``
    links_norms = True

    def set_output_scale(self, scale):
        """``scale`` (float32 [hidden]) multiplies what the mixer adds."""
        self.o.out_scale = scale

    def kernel_units(self):
        return kernels.gemm_units(self.compute) + [("recurrent", ())]

    def cache_needs(self):
        return [StateNeed((self.heads, kernels.matrix_memory_floats(self.dim, self.vdim))),
                StateNeed((self.heads, kernels.matrix_memory_aux_floats(self.dim, self.vdim)))]

    def weight_bytes(self):
        return self.proj.bytes() + self.o.bytes() + 4 * self.norm.numel()

    def forward(self, ctx, h, residual, caches, writes_cache=True, then_norm=None):
        if not writes_cache:
            raise ValueError("matrix_memory: a recurrent mixer cannot run on another layer's state")
        state, aux = caches
        hd, hv, nh = self.hd, self.hv, self.heads
        p = self.proj(h, out_dtype=torch.float32)
        t = p.shape[0]
        at = 2 * (hd + hv)
        y = torch.empty((t, hv), dtype=torch.float32, device=p.device)
        kernels.matrix_memory(p[:, :hd], p[:, hd:2 * hd], p[:, 2 * hd:2 * hd + hv], p[:, at:at + nh], p[:, at + nh:at + 2 * nh],
                              state, aux, ctx.cu_seqlens, ctx.seq_slot, y, nh, self.dim, self.vdim, self.cap,
                              float(self.dim) ** -0.5)
        out = torch.empty((t, hv), dtype=self.act_dtype, device=p.device)
        kernels.gated_group_norm(y, p[:, 2 * hd + hv:at], self.norm, out, self.vdim, self.eps, False, self.out_scale, "sigmoid")
        return self.o.add_into(out, residual, then_norm)


register_part("mixer", "matrix_memory", MatrixMemory)

"""A layer's own input for each token: behind its sublayers a layer adds a vector made of the token's row in a second embedding
table and gated by the stream,
    e = table[token, i * dim : (i + 1) * dim]                     the columns of layer i; one table serves all layers
    y = W_proj (gelu_tanh(W_gate x) * e);   x <- x + norm_w * y * rsqrt(mean(y^2) + eps)
x is the residual stream itself, read in the compute dtype, after everything that the layer's sublayers leave in it. The norm and the
add run in the launch of the next norm (``NormedDelta``); for decode rows the gate and the table's row are applied in the
epilogue of the gate's product.

Tensor names below the part's prefix: gate, proj, norm. The table belongs to the model, which passes it on with ``set_table``.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import NormedDelta, Part
from .linear import linear
from . import linear as linear_mod
from .norm import RMSNorm, add_to_stream


class TokenSideInput(Part):
    capturable = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.hidden = int(params["hidden_size"])
        self.dim = int(params["dim"])
        self.index = int(params["index"])                     # the layer's place in the table
        self.pad = -(-self.dim // 8) * 8                      # rows of 16-byte multiples for the products
        self.norm = RMSNorm({"size": self.hidden, "eps": params["eps"], "weight_name": "norm"}, dtype, device)
        self.gate = self.proj = self.table = None

    def weight_shapes(self):
        return {"gate": (self.dim, self.hidden), "proj": (self.hidden, self.dim), **self.norm.weight_shapes()}

    def keeps_dtype(self, name):
        return name == "norm"

    def load_weights(self, tensors):
        gate, proj = tensors["gate"], tensors["proj"]
        if self.pad > self.dim:
            more = self.pad - self.dim
            gate = torch.cat([gate, torch.zeros(more, self.hidden, dtype=gate.dtype, device=gate.device)], 0)
            proj = torch.cat([proj, torch.zeros(self.hidden, more, dtype=proj.dtype, device=proj.device)], 1)
        self.gate, self.proj = gate.contiguous(), proj.contiguous()
        self.norm.load_weights({"norm": tensors["norm"]})

    def set_table(self, table: torch.Tensor) -> None:
        """``table`` [vocab, layers * dim] in the compute dtype."""
        self.table = table[:, self.index * self.dim:(self.index + 1) * self.dim]

    def kernel_files(self, page_size):
        return ("stream_add", "embedding") + (("gemm_f32",) if self.dtype == torch.float32 else ("gemm_skinny", "gemm_rows", "gemm_tc05"))

    def forward(self, resid, delta, ctx) -> NormedDelta:
        T = resid.shape[0]
        x = ctx.buf("block_x", (T, self.hidden), self.dtype)
        add_to_stream(resid, delta, x)
        g = ctx.buf("side_gate", (T, self.pad), self.dtype)
        if linear_mod.USE_SKINNY and ops.gemm_skinny_ok(x, self.gate, g):
            ops.gemm_skinny_token_gate(x, self.gate, g, ctx.tokens, self.table, self.dim, checked=True)
        else:
            linear(x, self.gate, g, ctx.status)
            ops.token_gate(g, ctx.tokens, self.table, g)
        y = ctx.buf("side_delta", (T, self.hidden), self.dtype)
        linear(g, self.proj, y, ctx.status)
        return NormedDelta(y, self.norm)

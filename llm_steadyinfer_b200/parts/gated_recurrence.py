"""Recurrent block with a real-gated linear recurrence: two branches of one width, one of which runs through a short causal convolution
and a recurrence per channel, the other gates the result.

Per row x, with width W in ``blocks`` equal parts:
    y = gelu_tanh(W_y x + b_y);   u = conv(W_x x + b_x) + b_c             ``conv_taps`` taps per channel, the last one the current token's
    r = sigmoid(R_b u_b + b_r),  i = sigmoid(I_b u_b + b_i)               per part b, square matrices
    a = exp(-8 r softplus(lam));   S <- a S + sqrt(1 - a^2) i u           per channel, fp32, zero at the start
    out = W_o (S * y)
A request's state is one fp32 vector per slot: ``[S: W | the convolution's last taps - 1 inputs]``; kernels start a portion from it and
leave the next portion's behind. The gates' products take u in the compute dtype with fp32 sums; the gates, the decay and the
recurrence are fp32 in both precisions. Both gates of all parts are one launch: batched weight-streaming products for decode
rows, else the grouped product of the routed feed-forward with a part as a group.

Tensor names below the part's prefix: y[.b], x[.b], conv[.b], ra[.b], ri[.b], lam, o.
"""
from __future__ import annotations

import numpy as np
import torch

from ..csrc import ops
from .base import Mixer, StateNeed, register_mixer
from .linear import linear
from . import linear as linear_mod
from .step_rows import portions, row_kinds

DECAY_RATE = 8.0


class GatedRecurrence(Mixer):
    capturable = True

    def __init__(self, params, dtype, device, position=None):
        super().__init__(params, dtype, device, position)
        p = params
        self.hidden = int(p["hidden_size"])
        self.W = int(p["width"])
        self.blocks = int(p["blocks"])
        self.taps = int(p["conv_taps"])
        if self.W % self.blocks:
            raise ValueError(f"gated_recurrence: width {self.W} does not split into {self.blocks} parts")
        if self.taps < 1:
            raise ValueError(f"gated_recurrence: {self.taps} convolution taps")
        self.bs = self.W // self.blocks
        self.bs_pad = -(-self.bs // 8) * 8                        # rows of 16-byte multiples for the gates' products
        self.head_width = self.W
        self.x_off = -(-self.W // 8) * 8                          # the x branch's columns of the stacked projection
        self.conv_off = -(-self.W // 4) * 4
        self.input_weight = self.output_weight = self.w_gates = None
        self.y_bias = self.x_bias = self.taps_w = self.conv_bias = self.r_bias = self.i_bias = self.rate = None

    def weight_shapes(self):
        d, W, B, b = self.hidden, self.W, self.blocks, self.bs
        return {"y": (W, d), "y.b": (W,), "x": (W, d), "x.b": (W,), "conv": (W, self.taps), "conv.b": (W,), "ra": (B, b, b), "ra.b": (B, b),
                "ri": (B, b, b), "ri.b": (B, b), "lam": (W,), "o": (d, W)}

    def keeps_dtype(self, name):
        return name.endswith(".b") or name in ("conv", "lam")

    def norm_like(self, name):
        return False

    def load_weights(self, t):
        rows = []
        for n in ("y", "x"):
            rows.append(t[n])
            if self.x_off > self.W:
                rows.append(torch.zeros(self.x_off - self.W, self.hidden, dtype=t[n].dtype, device=t[n].device))
        self.input_weight = torch.cat(rows, 0).contiguous()
        self.output_weight = t["o"].contiguous()
        gates = torch.cat([t["ra"], t["ri"]], 1)                  # [blocks, 2 bs, bs]
        if self.bs_pad > self.bs:
            gates = torch.nn.functional.pad(gates, (0, self.bs_pad - self.bs))
        self.w_gates = gates.contiguous()
        f32 = lambda n: t[n].float().reshape(-1).contiguous()
        self.y_bias, self.x_bias, self.conv_bias = f32("y.b"), f32("x.b"), f32("conv.b")
        self.r_bias, self.i_bias = f32("ra.b"), f32("ri.b")
        self.taps_w = t["conv"].float().t().contiguous()
        self.rate = (DECAY_RATE * torch.nn.functional.softplus(t["lam"].double())).float().contiguous()

    def state_need(self):
        return StateNeed((self.conv_off + -(-(self.taps - 1) * self.W // 4) * 4,), torch.float32)

    def streams_first(self, rows):
        return self.input_weight if self.dtype == torch.bfloat16 and rows <= ops.SKINNY_MAX_ROWS else None

    def kernel_files(self, page_size):
        return ("qkv_conv", "gated_linear", "moe") + (("gemm_f32",) if self.dtype == torch.float32 else ("gemm_skinny", "gemm_rows", "gemm_tc05"))

    def _few(self, rows: int) -> bool:
        return self.dtype == torch.bfloat16 and linear_mod.USE_SKINNY and rows <= ops.SKINNY_MAX_ROWS

    def prepare(self, ctx, cache):
        key = ("gated_recurrence", self.blocks)
        if key not in ctx.plans and not self._few(ctx.num_tokens):        # first row of every part among the stacked rows
            ctx.plans[key] = ctx.upload_ints(f"gated_parts_{self.blocks}", np.arange(self.blocks + 1, dtype=np.int32) * ctx.num_tokens)

    def forward_heads(self, x, ctx, cache, out, scale: float = 1.0, proj=None):
        """``scale * S * y`` into ``out`` [T, W] (a view with a row stride): everything but W_o."""
        T, W, B = x.shape[0], self.W, self.blocks
        if proj is None:
            proj = ctx.buf("gated_proj", (T, self.input_weight.shape[0]), self.dtype)
            linear(x, self.input_weight, proj, ctx.status)
        u = ctx.buf("gated_u", (T, W), torch.float32)
        parts = ctx.buf("gated_parts", (B, T, self.bs_pad), self.dtype)       # columns beyond bs meet zero weights and stay finite
        ops.conv_rows(proj[:, self.x_off:self.x_off + W], self.x_bias, self.taps_w, cache.state[:, self.conv_off:], ctx.positions,
                      ctx.row_seq, ctx.q_start, ctx.ctx_len, ctx.slots, ctx.seq_slots, 0, 0, B, self.bs, self.bs, u,
                      out_bias=self.conv_bias, copy=parts, portions=portions(ctx), status=ctx.status)
        z = ctx.buf("gated_z", (B, T, 2 * self.bs), torch.float32)
        if self._few(T):
            ops.gemm_skinny_batched(parts, self.w_gates, z)
        else:
            ops.moe_gemm(parts.view(B * T, self.bs_pad), None, self.w_gates, z.view(B * T, 2 * self.bs),
                         ctx.plans[("gated_recurrence", B)], status=ctx.status)
        ops.gated_linear(u, z, self.r_bias, self.i_bias, self.rate, proj[:, :W], self.y_bias, cache.state, out, ctx.q_start, ctx.ctx_len,
                         ctx.slots, ctx.seq_slots, scale, row_kinds(ctx))

    def forward(self, x, ctx, cache):
        T = x.shape[0]
        heads = ctx.buf("gated_heads", (T, self.x_off), self.dtype)[:, :self.W]
        self.forward_heads(x, ctx, cache, heads)
        out = ctx.buf("delta", (T, self.hidden), self.dtype)
        linear(heads, self.output_weight, out, ctx.status)
        return out


register_mixer("gated_recurrence", GatedRecurrence)

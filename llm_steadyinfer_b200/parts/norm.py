"""Norms of the residual stream.

RMSNorm part: ``out = weight * h * rsqrt(mean(h^2) + eps)`` with ``h = resid + delta``
written back to the fp32 residual stream. Formula of the reference's
``row_rmsnorm_f32_dim`` (src/source/op/kernels/cuda/rmsnorm_kernel.cu:8-60), whose eps is a
constant in the kernel; here it is a parameter of the part. With ``scalar`` the checkpoint holds one number
for all coordinates (a tensor without dimensions), which is spread over the width when the weights are loaded.
With ``offset`` c the checkpoint's vector is stored around zero and the norm multiplies by ``c + weight`` (summed in fp32
when the weights are loaded, and kept in fp32). With ``gain`` g the result is multiplied by g (the weight is, in fp32, when it
is loaded).

Dynamic tanh part (kind "dynamic_tanh"): ``out = tanh(alpha * h) * weight + bias``, entry by entry, without mean or variance; ``alpha`` is
one learned number, and all three are kept in fp32 (tensor names below the part's prefix: the vector's, ``.b``, ``.alpha``).

A norm takes whatever a block leaves to be added (a plain result, one that is still to pass a norm behind its sublayer, the
results of two sublayers): ``add_to_stream`` does it for norms of any kinds; two RMS norms have a kernel of their own.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from .base import Norm, NormedDelta, SummedDelta, register_norm


class RMSNorm(Norm):
    capturable = True
    takes_ahead = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.name = params.get("weight_name", "weight")      # "" where the checkpoint names the vector by the prefix alone
        self.scalar = bool(params.get("scalar", False))     # one number for all coordinates
        self.offset = float(params.get("offset", 0.0))      # added to the stored vector
        self.gain = float(params.get("gain", 1.0))          # what the result is multiplied by
        self.weight: Optional[torch.Tensor] = None
        self._weight32: Optional[torch.Tensor] = None

    def weight_shapes(self):
        return {self.name: () if self.scalar else (self.size,)}

    def keeps_dtype(self, name: str) -> bool:
        return True

    def load_weights(self, tensors):
        w = tensors[self.name]
        if self.offset:
            w = w.float() + self.offset
        if self.gain != 1.0:
            w = w.float() * self.gain
        self.weight = (w.reshape(1).expand(self.size) if self.scalar else w).contiguous()

    def norm_like(self, name):
        return not self.offset                       # a vector stored around zero is drawn around zero

    def kernel_files(self, page_size):
        return ("norm",)

    def forward(self, resid, delta, out, rows=None, ahead=None):
        if isinstance(delta, NormedDelta) and not isinstance(delta.norm, RMSNorm):
            add_to_stream(resid, delta, out, self, rows)
        elif isinstance(delta, NormedDelta):         # the sublayer before has a norm of its own behind it
            ops.add_norm(resid, delta.x, self.weight, self.eps, out, rows=rows, delta_weight=delta.norm.weight,
                         delta_eps=delta.norm.eps, delta_bias=delta.bias)
        elif isinstance(delta, SummedDelta):         # two sublayers side by side: both join the stream here
            ops.add_rmsnorm(resid, delta.a, self.weight, self.eps, out, rows=rows, ahead=ahead, delta2=delta.b)
        else:
            ops.add_rmsnorm(resid, delta, self.weight, self.eps, out, rows=rows, ahead=ahead)

    def forward_streams(self, resid, delta, connections, out, rows=None, ahead=None):
        c = delta.connections
        ops.stream_norm(resid if delta.spread is None else delta.spread, self.weight, self.eps, out,
                        dst=resid if rows is None and delta.y is not None else None, y=delta.y,
                        mix=None if delta.y is None else c.mix, write=None if delta.y is None else c.write,
                        read=None if connections is None else connections.read, rows=rows, ahead=ahead, streams=resid.shape[1])

    def add(self, resid, delta: NormedDelta, extra=None, vec=None):
        """``resid += norm(delta) (+ extra) (+ vec)`` with no norm of the stream behind it."""
        ops.add_norm(resid, delta.x, delta_weight=delta.norm.weight, delta_eps=delta.norm.eps, delta_bias=delta.bias,
                     extra=extra, vec=vec)

    def normalize(self, x, out=None):
        ops.rmsnorm_rows(x, self.weight, self.eps, out)

    def plain(self, x):
        return x * torch.rsqrt((x * x).mean(-1, keepdim=True) + self.eps) * self.weight.float()

    def stream_norm(self):
        if self._weight32 is None:
            self._weight32 = self.weight.float().contiguous()
        return ("rms", self._weight32, self.eps)


register_norm("rmsnorm", RMSNorm)


class DynamicTanh(Norm):
    capturable = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.size = int(params["size"])
        self.name = params.get("weight_name", "weight")
        self.bias_name = params.get("bias_name", ".b")
        self.alpha_name = params.get("alpha_name", ".alpha")
        self.gain = float(params.get("gain", 1.0))          # what the result is multiplied by
        self.weight = self.bias = None
        self.alpha = 1.0

    def weight_shapes(self):
        return {self.name: (self.size,), self.bias_name: (self.size,), self.alpha_name: ()}

    def keeps_dtype(self, name):
        return True

    def norm_like(self, name):
        return name != self.bias_name

    def load_weights(self, tensors):
        self.weight = (tensors[self.name].float() * self.gain).contiguous()
        self.bias = (tensors[self.bias_name].float() * self.gain).contiguous()
        self.alpha = float(tensors[self.alpha_name].float().item())

    def kernel_files(self, page_size):
        return ("stream_add",)

    def forward(self, resid, delta, out, rows=None):
        add_to_stream(resid, delta, out, self, rows)

    def plain(self, x):
        return torch.tanh(self.alpha * x) * self.weight + self.bias

    def stream_norm(self):
        return ("tanh", self.weight, self.bias, self.alpha)


register_norm("dynamic_tanh", DynamicTanh)


def add_to_stream(resid, delta, out=None, norm: Optional[Norm] = None, rows=None) -> None:
    """``resid += delta``, whatever form it has, and ``out = norm(resid)`` (``norm`` None: the stream as it is, in out's dtype)."""
    if isinstance(delta, SummedDelta):
        ops.stream_add(resid, delta.a)
        delta = delta.b
    if isinstance(delta, NormedDelta):
        ops.stream_add(resid, delta.x, delta.norm.stream_norm(), delta.bias, out, None if norm is None else norm.stream_norm(), rows)
    else:
        ops.stream_add(resid, delta, out=out, norm=None if norm is None else norm.stream_norm(), rows=rows)

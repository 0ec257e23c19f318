"""Connections of a sublayer to a residual stream kept in several copies ("streams").

A sublayer reads one row made of all S streams and writes its result back into all of them, with learned numbers:
    u = sum_s read[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + write[t] y     (all from the old x_s)
They are a part of their own beside the sublayer's norm (tensor names below the part's prefix: ``in`` [S], ``out`` [S],
``mix`` [S, S], [from, to]), kept in fp32. The arithmetic runs in the launch between two sublayers
(``Norm.forward_streams``), which writes the streams after one sublayer, reads for the next and normalises.
"""
from __future__ import annotations

import torch

from .base import Part


class StreamConnections(Part):
    capturable = True

    def __init__(self, params, dtype, device):
        super().__init__(params, dtype, device)
        self.streams = int(params["streams"])
        if self.streams < 1:
            raise ValueError(f"stream connections: {self.streams} streams")
        self.read = self.write = self.mix = None

    def weight_shapes(self):
        S = self.streams
        return {"in": (S,), "out": (S,), "mix": (S, S)}

    def keeps_dtype(self, name):
        return True

    def norm_like(self, name):
        return name != "mix"

    def identity_like(self, name):
        return name == "mix"

    def load_weights(self, tensors):
        self.read = tensors["in"].float().contiguous()
        self.write = tensors["out"].float().contiguous()
        self.mix = tensors["mix"].float().contiguous()

    def kernel_files(self, page_size):
        return ("streams",)

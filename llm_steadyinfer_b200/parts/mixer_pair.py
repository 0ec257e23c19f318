"""Two mixers side by side: both read the same input, and the block gets ``left_scale * left(x) + right_scale * right(x)``.

The two are registered mixer kinds of their own, built from ``params["left"]`` / ``params["right"]`` = ``{"kind": ..,
"params": .., "position": {"kind": .., "params": ..} or None}``; their checkpoint tensors lie below ``left.`` and
``right.`` (``prefixes`` overrides). Between them they may ask for one paged cache, which the pair passes on as its own need; where
both keep state, the pair's slot holds the left one's, then the right one's (on a 16-byte boundary), and each sees its own part.

Both kinds must offer the pair their result *before* the output projection: ``forward_heads(x, ctx, cache, out, scale)``
writes the scaled, gated heads into the strided view ``out`` [T, head_width], and ``output_weight`` is the projection
[hidden, head_width]. The pair stacks the two projections along k at load, so that one product over
``[scale_l * heads_l | scale_r * heads_r]`` gives the weighted sum: each scale is applied in fp32 where the heads are
formed, and the two results are added in the product's fp32 sums, never as rounded tensors. A kind that says
``folds_head_scale`` takes its scale as the parameter ``head_scale`` instead.
Where both kinds offer their input projection as one matrix (``input_weight`` [rows, hidden], rows a multiple of 8) the pair stacks
these as well and passes each its columns of the one product (``forward_heads(..., proj=)``).
"""
from __future__ import annotations

import dataclasses

import torch

from ..csrc import ops
from .base import Mixer, StateNeed, mixer_class, position_class, register_mixer
from .linear import linear


class MixerPair(Mixer):
    def __init__(self, params, dtype, device, position=None):
        super().__init__(params, dtype, device, position)
        self.hidden = int(params["hidden_size"])
        self.scales = (float(params.get("left_scale", 1.0)), float(params.get("right_scale", 1.0)))
        self.prefixes = tuple(params.get("prefixes") or ("left.", "right."))
        self.subs = []
        for side in ("left", "right"):
            sp = params[side]
            pos = sp.get("position")
            pos = None if pos is None else position_class(pos["kind"])(pos["params"], dtype, device)
            cls, sparams = mixer_class(sp["kind"]), dict(sp["params"])
            if getattr(cls, "folds_head_scale", False):
                sparams["head_scale"] = self.scales[len(self.subs)]
            sub = cls(sparams, dtype, device, position=pos)
            if not hasattr(sub, "forward_heads") or not hasattr(sub, "head_width"):
                raise ValueError(f"mixer_pair: mixer kind {sp['kind']!r} does not offer its heads before the output projection")
            self.subs.append(sub)
        caches = [s.cache_need() for s in self.subs if s.cache_need() is not None]
        states = [s.state_need() for s in self.subs]
        if len(caches) > 1:
            raise ValueError("mixer_pair: the two mixers may ask for one paged cache between them")
        self.scales = tuple(1.0 if getattr(type(s), "folds_head_scale", False) else c for s, c in zip(self.subs, self.scales))
        self._cache_need = caches[0] if caches else None
        self._state_need = next((s for s in states if s is not None), None)
        self._state_parts = None                     # (first entry, entries) of each mixer's state where both have one
        if all(s is not None for s in states):
            if any(len(s.shape) != 1 for s in states) or states[0].dtype != states[1].dtype:
                raise ValueError("mixer_pair: two states go together as vectors of one dtype")
            n0, n1 = int(states[0].shape[0]), int(states[1].shape[0])
            at = -(-n0 // 4) * 4
            self._state_parts = ((0, n0), (at, n1))
            self._state_need = StateNeed((-(-(at + n1) // 4) * 4,), states[0].dtype)
        self._views = {}                             # a state tensor's address -> each mixer's part of it
        self.widths = tuple(int(s.head_width) for s in self.subs)
        self.w_o = self.w_in = None
        self._columns = None

    @property
    def capturable(self):
        return all(s.capturable for s in self.subs)

    def weight_shapes(self):
        return {p + n: shape for p, s in zip(self.prefixes, self.subs) for n, shape in s.weight_shapes().items()}

    def _owner(self, name):
        for p, s in zip(self.prefixes, self.subs):
            if name.startswith(p) and name[len(p):] in s.weight_shapes():
                return s, name[len(p):]
        raise KeyError(name)

    def keeps_dtype(self, name):
        s, n = self._owner(name)
        return s.keeps_dtype(n)

    def norm_like(self, name):
        s, n = self._owner(name)
        return s.norm_like(n)

    def load_weights(self, tensors):
        for p, s in zip(self.prefixes, self.subs):
            s.load_weights({n: tensors[p + n] for n in s.weight_shapes()})
        # one output product for both: [hidden, width_l + width_r], k padded to a multiple of 8 for the kernels' 16-byte rows
        ws = [s.output_weight for s in self.subs]
        k = sum(self.widths)
        self.k_pad = -(-k // 8) * 8
        if self.k_pad > k:
            ws.append(torch.zeros(self.hidden, self.k_pad - k, dtype=ws[0].dtype, device=ws[0].device))
        self.w_o = torch.cat(ws, 1).contiguous()
        for s in self.subs:
            s.output_weight = None                   # the stacked matrix is the one that is used
        ins = [getattr(s, "input_weight", None) for s in self.subs]
        if all(w is not None and w.shape[0] % 8 == 0 for w in ins):
            self.w_in = torch.cat(ins, 0).contiguous()
            n0 = int(ins[0].shape[0])
            self._columns = ((0, n0), (n0, int(self.w_in.shape[0])))
            for s in self.subs:
                s.input_weight = None

    def cache_need(self):
        return self._cache_need

    def state_need(self):
        return self._state_need

    def streams_first(self, rows):
        if self.w_in is not None:
            return self.w_in if self.dtype == torch.bfloat16 and rows <= ops.SKINNY_MAX_ROWS else None
        return self.subs[0].streams_first(rows)

    def kernel_files(self, page_size):
        names = set()
        for s in self.subs:
            names.update(s.kernel_files(page_size))
        return tuple(sorted(names))

    def _caches(self, cache):
        """The layer's cache as each mixer sees it."""
        if self._state_parts is None:
            return (cache, cache)
        key = cache.state.data_ptr()
        views = self._views.get(key)
        if views is None:
            views = self._views[key] = tuple(cache.state[:, a:a + n] for a, n in self._state_parts)
        return tuple(dataclasses.replace(cache, state=v) for v in views)

    def prepare(self, ctx, cache):
        for s in self.subs:
            s.prepare(ctx, cache)

    def forward(self, x, ctx, cache):
        T = x.shape[0]
        heads = ctx.buf("pair_heads", (T, self.k_pad), self.dtype)       # the padding columns stay zero
        proj = None
        if self.w_in is not None:
            proj = ctx.buf("pair_proj", (T, self.w_in.shape[0]), self.dtype)
            linear(x, self.w_in, proj, ctx.status)
        at = 0
        for i, (s, w, scale, c) in enumerate(zip(self.subs, self.widths, self.scales, self._caches(cache))):
            if proj is None:
                s.forward_heads(x, ctx, c, heads[:, at:at + w], scale)
            else:
                a, b = self._columns[i]
                s.forward_heads(x, ctx, c, heads[:, at:at + w], scale, proj=proj[:, a:b])
            at += w
        out = ctx.buf("pair_delta", (T, self.hidden), self.dtype)     # a buffer of its own: it may live beside a feed-forward's
        linear(heads, self.w_o, out, ctx.status)
        return out


register_mixer("mixer_pair", MixerPair)

"""Attention mixer: grouped-query causal attention over the paged cache, optional window, optional learned bias by
distance, a value size that may differ from the key size.

Per row: q, k, v from one stacked projection [ (H + 2 KV) * hs, d ] (the reference stacks
them too, src/source/model/llama3.cpp:434-498, but then reads the output with the wrong row
stride, llama3.cpp:1009-1019; every consumer here takes the row stride); rotation of q and k
and the store of k, v into the sequence's pages; softmax(scale * q . K) V over cache
positions up to the row's own (llama3.cpp:1048-1067); output projection (llama3.cpp:1136-1140).

Options beyond the reference's block, all parameters of the part:
``value_dim``      size of a value head (default ``head_dim``); the cache then keeps values of that size.
``distance_bias``  ``{"max_distance": D, "buckets": B or None, "name": tensor}``: a learned table [B, heads] whose row
                   ``bucket(i - j)`` is added to the scaled score of query i and key j. Distances below B/2 have a
                   row each; the other B - B/2 rows share the distances from B/2 to D on a logarithmic scale:
                   ``bucket(n) = min(B - 1, B/2 + floor(log(n / (B/2)) / log(D / (B/2)) * (B - B/2)))``. B None: the
                   checkpoint's tensor says how many rows there are. At load the table is spread out by distance
                   (one row for every n up to D), which is what the kernels index.
``names``          checkpoint names of the four matrices, ``{"q": .., "k": .., "v": .., "o": ..}``.
``values_are_keys`` the layer has no value projection: head g's value at a position is its key there, so the cache keeps keys
                   alone and the kernels read the values out of the key pages (a ``value_dim`` below ``head_dim``: the key's first entries).
``distance_slopes`` ``{"base": b, "exponent": e}``: ``slope_h * (i - j)`` with ``slope_h = b^(e (h + 1) / heads)`` is taken off
                   the scaled score of query i and key j (a penalty in proportion to the distance, steeper for the first heads).
``query_temperature`` ``{"coef": c, "every": n}``: the query at position p is multiplied by ``1 + c ln(floor((p + 1) / n) + 1)``
                   (applied by the attention kernels to the row's scale, in fp32).
``output_gate``    name of a matrix [heads * value_dim, hidden]: the heads' results are multiplied entry by entry with
                   ``sigmoid(W_g x)`` before the output projection; its rows are stacked behind q, k, v in one product, and the
                   attention kernels apply the gate when they store their results.
``biases``         the projections of q, k and v have biases (tensor names: the matrix's + ``bias_suffix``).
``conv_taps``      K: every channel of q, k and v passes a causal convolution over time of K taps (tensor names: the matrix's +
                   ``conv_suffix``, [channels, K], the last tap the current token's); the last K - 1 projected values of a request
                   are its state.
``qk_norm``        ``{"eps": e}``: every query and key head is scaled to a root mean square of one (after the convolution).
``rot_interleaved`` the layer's rotary position encoding turns neighbouring pairs (2i, 2i + 1) of its first entries (in the launch behind the
                   projection, between convolution and norm).
``head_scale``     the heads' results are multiplied by it (their values are, in fp32, before they are stored).
``sink_score``     a number s: exp(s) joins every row's softmax denominator once, without a value.
``chunk``          positions fall into runs of so many, counted from position 0; a query sees keys of its own run alone.
``own_keys``       False: the layer has no key and value projections and reads the cache of another one (its spec's
                   ``cache_from``), whose keys lie there as that layer stored them.
With any option but ``names`` the mixer runs its general form. Biases, convolution and norm are one launch behind the stacked
projection (``qkv_conv.cu``), which also stores keys and values. The attention itself: where scores are plain but for the sink
and the chunk and the sizes are ones that the fast kernels take (multiples of 8 up to 128), decode rows go to
``attention_tma.cu`` and prompt portions to ``attention_tc05.cu`` as in the reference's block; else the general kernels
(``attention_general.cu`` in 32-bit, ``attention_flex.cu`` on the tensor cores in bfloat16). Sequences that bring a full work item of
rows to a bfloat16 step go to the tcgen05 prompt kernel (``attention_tc05.cu``) where its layout fits (key size 64 or 128,
values of the same size or the keys themselves, no bias table): it takes slopes, temperature, gate, chunks and sink as well.
"""
from __future__ import annotations

import math

import numpy as np
import torch

from ..csrc import ops
from .base import CacheNeed, Mixer, StateNeed, first_visible_key, register_mixer
from . import flex_plan
from .step_rows import portions
from . import linear as linear_mod
from .linear import linear


USE_TENSOR_CORES = True      # bf16 only; False sends bf16 through the plain kernel as well
USE_TMA = True               # decode tiles by TMA where the layout allows
USE_TC05 = True              # prompt portions on tcgen05 where the layout allows
FUSE_ROPE = True             # few rows (decode): rotation and cache store in the epilogue of the q/k/v product
DECODE_BLOCKS_PER_SM = 2     # decode attention blocks that one multiprocessor holds at once
MAX_SPLITS = 32
MIN_TILES_PER_SPLIT = 2      # a split covers at least this many 64-key tiles


class Attention(Mixer):
    adds_into_residual = True
    folds_head_scale = True          # a pair of mixers passes this side's scale as a parameter

    def __init__(self, params, dtype, device, position=None):
        super().__init__(params, dtype, device, position)
        self.hidden = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.KV = int(params["num_kv_heads"])
        self.hs = int(params["head_dim"])
        self.scale = float(params["scale"])
        self.window = params.get("window") or None
        if self.H % self.KV:
            raise ValueError(f"attention: {self.H} heads are not a multiple of {self.KV} kv heads")
        self.vs = int(params.get("value_dim") or self.hs)
        self.names = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight"}
        self.names.update(params.get("names") or {})
        self.bias_spec = params.get("distance_bias") or None
        if self.bias_spec is not None:
            self.bias_name = self.bias_spec.get("name", "distance_bias")
            self.bias_rows = self.bias_spec.get("buckets")
            self.bias_max = float(self.bias_spec["max_distance"])
        self.own_v = not bool(params.get("values_are_keys", False))
        if not self.own_v and self.vs > self.hs:
            raise ValueError(f"attention: values that are the keys have at most the keys' size {self.hs}, found value_dim {self.vs}")
        sl = params.get("distance_slopes") or None
        self.slopes = None               # fp32 [H] on the device
        if sl is not None:
            base, expo = float(sl["base"]), float(sl["exponent"])
            self.slopes = torch.tensor([base ** (expo * (h + 1) / self.H) for h in range(self.H)], dtype=torch.float64) \
                .to(torch.float32).to(device)
        qt = params.get("query_temperature") or None
        self.q_temp = None if qt is None else (float(qt["coef"]), qt["every"])
        self.gate_name = params.get("output_gate") or None
        self.chunk = params.get("chunk") or None
        self.sink_score = params.get("sink_score")
        self.sink = None                 # fp32 [H] on the device
        if self.sink_score is not None:
            self.sink = torch.full((self.H,), float(self.sink_score), dtype=torch.float32, device=device)
        self.biases = bool(params.get("biases", False))
        self.bias_suffix = params.get("bias_suffix", ".bias")
        self.taps = int(params.get("conv_taps") or 1)
        self.has_conv = params.get("conv_taps") is not None
        self.conv_suffix = params.get("conv_suffix", ".conv")
        qkn = params.get("qk_norm") or None
        self.qk_norm = qkn is not None
        self.qk_eps = float(qkn["eps"]) if self.qk_norm else 0.0
        self.own_keys = bool(params.get("own_keys", True))
        self.rot_interleaved = bool(params.get("rot_interleaved", False))
        self.head_scale = float(params.get("head_scale", 1.0))
        # a launch behind the projection
        self.prepared = self.biases or self.has_conv or self.qk_norm or not self.own_keys or self.rot_interleaved or self.head_scale != 1.0
        self.head_width = self.H * self.vs
        # scores that the fast kernels know: q . k times the scale, a window or chunks, a sink
        self.plain_scores = (self.bias_spec is None and self.own_v and self.slopes is None and self.q_temp is None
                             and self.gate_name is None)
        self.general = not self.plain_scores or self.vs != self.hs or self.prepared or self.chunk is not None or self.sink is not None
        if self.hs > (1024 if self.general else 256) or self.vs > 1024:
            raise ValueError(f"attention: head_dim {self.hs} is not supported (at most 256, 1,024 in the general form)")
        if self.taps < 1:
            raise ValueError(f"attention: {self.taps} convolution taps")
        if self.prepared and (not self.own_v or self.gate_name is not None):
            raise ValueError("attention: values that are the keys and an output gate go without biases, convolution, query/key "
                             "norm and another layer's keys")
        self.rot = None                  # (inverse frequencies, entries turned), neighbouring pairs
        if self.prepared and position is not None and self.rot_interleaved:
            self.rot = position.rotary()
            if self.rot is None or self.rot[1] > self.hs or getattr(position, "magnitude", 1.0) != 1.0:
                raise ValueError("attention: rot_interleaved goes with a rotary position encoding of at most head_dim entries and magnitude 1")
        elif self.general and position is not None:
            raise ValueError("attention: the general form (a distance bias, slopes, a value size of its own, values that are "
                             "the keys, a query temperature, an output gate) goes without a position encoding, or with rot_interleaved")
        # columns of the stacked projection: q, k, v (if the layer has values of its own), the gate (if it has one)
        self.kv_cols = self.KV * (self.hs + (self.vs if self.own_v else 0)) if self.own_keys else 0
        self.channels = self.H * self.hs + self.kv_cols
        self.gate_off = self.H * self.hs + self.kv_cols
        self.proj_cols = -(-(self.gate_off + (self.H * self.vs if self.gate_name else 0)) // 8) * 8 if self.general else 0
        self.dist_bias = None            # fp32 [distances, H], made at load
        self.qkv = None
        self.qkv_bias = self.qkv_taps = None        # fp32 [channels], fp32 [taps, channels]
        self.o = None
        self.stacked = False             # True: a pair of mixers makes this layer's projections with the other side's

    def _projections(self):
        """(name, rows) of the matrices in the stacked projection that biases and convolutions belong to."""
        n = self.names
        out = [(n["q"], self.H * self.hs)]
        if self.own_keys:
            out.append((n["k"], self.KV * self.hs))
            if self.own_v:
                out.append((n["v"], self.KV * self.vs))
        return out

    def weight_shapes(self):
        n = self.names
        shapes = {n["o"]: (self.hidden, self.H * self.vs)}
        for name, rows in self._projections():
            shapes[name] = (rows, self.hidden)
            if self.biases:
                shapes[name + self.bias_suffix] = (rows,)
            if self.has_conv:
                shapes[name + self.conv_suffix] = (rows, self.taps)
        if self.gate_name:
            shapes[self.gate_name] = (self.H * self.vs, self.hidden)
        if self.bias_spec is not None:
            shapes[self.bias_name] = (self.bias_rows if self.bias_rows else -1, self.H)   # -1: as the checkpoint has it
        return shapes

    def keeps_dtype(self, name):
        if self.bias_spec is not None and name == self.bias_name:
            return True
        return any((self.biases and name == p + self.bias_suffix) or (self.has_conv and name == p + self.conv_suffix)
                   for p, _ in self._projections())

    def norm_like(self, name):
        return False

    def load_weights(self, tensors):
        n = self.names
        parts = [tensors[name] for name, _ in self._projections()] + ([tensors[self.gate_name]] if self.gate_name else [])
        stacked = lambda suffix: torch.cat([tensors[name + suffix].float() for name, _ in self._projections()], 0)
        if self.biases:
            self.qkv_bias = stacked(self.bias_suffix).contiguous()
        if self.has_conv:
            self.qkv_taps = stacked(self.conv_suffix).t().contiguous()
        elif self.prepared:                                  # one tap of one: the value itself
            self.qkv_taps = torch.ones(1, self.channels, dtype=torch.float32, device=parts[0].device)
        if self.head_scale != 1.0:                           # linear in the values: the taps that make them carry the scale
            self.qkv_taps[:, self.channels - self.KV * self.vs:] *= self.head_scale
        rows = sum(p.shape[0] for p in parts)
        if self.general and rows < self.proj_cols:           # rows of the product's result stay 16-byte aligned
            parts.append(torch.zeros(self.proj_cols - rows, self.hidden, dtype=parts[0].dtype, device=parts[0].device))
        self.qkv = torch.cat(parts, 0).contiguous()
        self.o = tensors[n["o"]].contiguous()
        if self.bias_spec is not None:
            self.dist_bias = spread_by_distance(tensors[self.bias_name].float(), self.bias_max)

    # what a pair of mixers stacks: the input projection's rows, the output projection
    @property
    def input_weight(self):
        return self.qkv if self.general else None

    @input_weight.setter
    def input_weight(self, w):
        self.qkv = w

    @property
    def output_weight(self):
        return self.o

    @output_weight.setter
    def output_weight(self, w):
        self.o = w

    def cache_need(self):
        if not self.own_v:
            return CacheNeed(self.KV, self.hs, self.window, 0, chunk=self.chunk)
        return CacheNeed(self.KV, self.hs, self.window, None if self.vs == self.hs else self.vs, chunk=self.chunk)

    def state_need(self):
        if self.taps == 1:
            return None
        # rows of a multiple of four entries: a slot starts on a 16-byte boundary
        return StateNeed((-(-(self.taps - 1) * self.channels // 4) * 4,), torch.float32)

    @property
    def capturable(self):
        """The step's work lists are made in ``prepare``; a position encoding applied through its
        unfused hook decides for itself."""
        return self.position is None or self.position.capturable

    def streams_first(self, rows):
        # few rows in bfloat16 go to the weight-streaming product, which reads every weight once
        return self.qkv if self.dtype == torch.bfloat16 and rows <= ops.SKINNY_MAX_ROWS else None

    def kernel_files(self, page_size):
        if self.general:
            names = ["qkv_conv"] if self.prepared else ["attention_general"]          # what stores keys and values
            if self.dtype == torch.float32:
                return tuple(names + ["attention_general", "gemm_f32"])
            names += ["gemm_skinny", "gemm_rows", "gemm_tc05"]
            if self.uses_fast(page_size):
                return tuple(names + ["attention_tma", "attention_tc05"])
            names.append("attention_flex")
            if self.hs % 8 or self.vs % 8:                                             # sizes that kernel does not take
                names.append("attention_general")
            if self.general_tc05_ok(page_size):
                names += ["attention_tma", "attention_tc05"]
            return tuple(names)
        names = ["rope_kv"] + (["gemm_f32"] if self.dtype == torch.float32 else ["gemm_skinny", "gemm_rows", "gemm_tc05"])
        if not self.uses_tensor_cores():
            return tuple(names + ["attention_ref"])
        names.append("attention_mma")
        if self.hs in (64, 128) and page_size in (8, 16, 32, 64):        # the layouts the TMA-fed kernels take
            names += ["attention_tma"] * bool(USE_TMA) + ["attention_tc05"] * bool(USE_TC05)
        return tuple(names)

    def forward(self, x, ctx, cache, resid=None):
        if self.general:
            return self.forward_general(x, ctx, cache)
        T = x.shape[0]
        H, KV, hs = self.H, self.KV, self.hs
        qkv = ctx.buf("attn_qkv", (T, (H + 2 * KV) * hs), self.dtype)
        rot = self.position.rotary() if self.position is not None else None
        if (FUSE_ROPE and linear_mod.USE_SKINNY and rot is not None and rot[1] == hs and hs % 16 == 0
                and self.dtype == torch.bfloat16 and ops.gemm_skinny_ok(x, self.qkv, qkv)):
            # a decode step: one kernel for the projection, the rotation and the store into the pages
            ops.gemm_skinny_qkv_rope(x, self.qkv, qkv, ctx.positions, ctx.row_seq, rot[0], cache.block_table,
                                     cache.k if cache.writes else None, cache.v if cache.writes else None,
                                     cache.page_size, ctx.seq_slots, H, KV, hs, status=ctx.status)
            attn = ctx.buf("attn_out", (T, H * hs), self.dtype)
            self.attend(qkv[:, :H * hs], cache, ctx, attn)
            out = ctx.buf("delta", (T, self.hidden), self.dtype)
            linear(attn, self.o, out, ctx.status)
            return out
        linear(x, self.qkv, qkv, ctx.status)
        if self.position is not None and rot is None:
            q3 = qkv[:, :H * hs].view(T, H, hs)
            k3 = qkv[:, H * hs:(H + KV) * hs].view(T, KV, hs)
            self.position.apply(q3, k3, ctx)
        inv_freq, rot_dim = rot if rot is not None else (None, 0)
        ops.rope_kv_write(qkv, ctx.positions, ctx.row_seq, inv_freq, rot_dim, cache.block_table,
                          cache.k if cache.writes else None, cache.v if cache.writes else None,
                          cache.page_size, ctx.seq_slots, H, KV, hs, status=ctx.status)
        attn = ctx.buf("attn_out", (T, H * hs), self.dtype)
        self.attend(qkv[:, :H * hs], cache, ctx, attn)
        if resid is not None and linear_mod.linear_into_residual(attn, self.o, resid, ctx.status):
            return None                                   # the output projection added itself into the stream
        out = ctx.buf("delta", (T, self.hidden), self.dtype)
        linear(attn, self.o, out, ctx.status)
        return out

    def general_tc05_ok(self, page_size: int) -> bool:
        """The general form's long portions on the tcgen05 prompt kernel: its layouts, and nothing it does not know."""
        return (USE_TC05 and self.bias_spec is None and self.vs == self.hs and (self.q_temp is None or self.q_temp[0] >= 0)
                and ops.attn_portion_tc05_ok(self.H, self.KV, self.hs, page_size))

    def _plan_general_tc05(self, ctx, page_size: int) -> dict:
        """Which sequences of the step go to the tcgen05 prompt kernel (those that bring at least one full item of rows),
        and their work items; the others are the general tensor-core kernel's."""
        key = ("attention_general_tc05", self.H, self.KV, self.hs, self.window, self.chunk)
        got = ctx.plans.get(key)
        if got is not None:
            return got
        out = {"skip": frozenset(), "all": False, "items": None}
        if ctx.seq_cap is None and self.general_tc05_ok(page_size):
            per = ops.attn_portion_tc05_tokens(self.H, self.KV)
            qs, cl = ctx.h_q_start, ctx.h_ctx_len
            chosen, items = [], []
            for s in range(ctx.num_seqs):
                row0, n = int(qs[s]), int(qs[s + 1] - qs[s])
                if n < per:
                    continue
                chosen.append(s)
                pos0 = int(cl[s]) - n
                items += [(s, row0 + b, min(per, n - b), pos0 + b) for b in range(0, n, per)]
            if chosen:
                out = {"skip": frozenset(chosen), "all": len(chosen) == ctx.num_seqs,
                       "items": ctx.upload_ints(f"attn_gen_tc05_{self._tag()}",
                                                np.asarray(items, dtype=np.int32)).view(-1, 4)}
        ctx.plans[key] = out
        return out

    def forward_general(self, x, ctx, cache):
        """Keys (and values of their own size, where the layer has them) into the pages as they are, or behind
        biases, convolution and norm; scores with the bias, the slopes and the query temperature, the sink in the denominator;
        the gate on the heads' results."""
        T = x.shape[0]
        attn = ctx.buf("attn_out", (T, self.H * self.vs), self.dtype)
        self.forward_heads(x, ctx, cache, attn)
        out = ctx.buf("delta", (T, self.hidden), self.dtype)
        linear(attn, self.o, out, ctx.status)
        return out

    def forward_heads(self, x, ctx, cache, attn, scale: float = 1.0, proj=None):
        """The heads' results into ``attn`` [T, heads * value_dim] (a view with a row stride): everything but the output projection.
        ``proj``: the input projection's result where the caller has made it."""
        if not self.general or scale != 1.0:
            raise ValueError("attention: heads before the output projection are the general form's; their scale is the parameter head_scale")
        T = x.shape[0]
        H, KV, hs, vs = self.H, self.KV, self.hs, self.vs
        qkv = proj
        if qkv is None:
            qkv = ctx.buf("attn_qkv", (T, self.proj_cols), self.dtype)
            linear(x, self.qkv, qkv, ctx.status)
        v_cache = cache.v if self.own_v else None
        q = qkv[:, :H * hs]
        if self.prepared:
            q = ctx.buf("attn_q", (T, H * hs), self.dtype)
            stores = cache.writes and self.own_keys
            kv = KV if self.own_keys else 0
            ops.qkv_conv(qkv, self.qkv_bias, self.qkv_taps, cache.state, ctx.positions, ctx.row_seq, ctx.q_start, ctx.ctx_len,
                         ctx.slots, cache.block_table, cache.k if stores else None, cache.v if stores else None, cache.page_size,
                         ctx.seq_slots, H, kv, kv, hs, vs, q, self.qk_norm, self.qk_eps, portions=portions(ctx), status=ctx.status,
                         inv_freq=None if self.rot is None else self.rot[0], rot_dims=0 if self.rot is None else self.rot[1])
        elif cache.writes:
            ops.kv_store(qkv, ctx.positions, ctx.row_seq, cache.block_table, cache.k, v_cache, cache.page_size,
                         ctx.seq_slots, H, KV, hs, vs if self.own_v else 0, status=ctx.status)
        gate = qkv[:, self.gate_off:self.gate_off + H * vs] if self.gate_name else None      # applied in the attention's epilogue
        if self.uses_fast(cache.page_size):
            self.attend(q, cache, ctx, attn)
        elif self.uses_flex():
            big = self._plan_general_tc05(ctx, cache.page_size)
            if not big["all"]:
                flex_plan.attend(flex_plan.plan(ctx, self.device, H, KV, hs, vs, self.own_v, self.window, skip=big["skip"],
                                                chunk=self.chunk),
                                 q, cache.k, v_cache, cache.block_table, attn, cache.page_size, ctx.seq_slots, H, KV,
                                 hs, vs, self.scale, self.window, dist_bias=self.dist_bias, sink=self.sink, status=ctx.status,
                                 slopes=self.slopes, q_temp=self.q_temp, gate=gate, chunk=self.chunk)
            if big["items"] is not None:
                ops.attn_portion_tc05(q, cache.k, v_cache, cache.block_table, big["items"], attn, cache.page_size,
                                      ctx.seq_slots, H, KV, hs, self.scale, self.window or 0, status=ctx.status,
                                      slopes=self.slopes, q_temp=self.q_temp, gate=gate, chunk=self.chunk or 0, sink=self.sink)
        else:
            ops.attention_general(q, cache.k, v_cache, cache.block_table, ctx.row_seq, ctx.positions, attn,
                                  cache.page_size, ctx.seq_slots, H, KV, hs, vs, self.scale, self.window or 0,
                                  dist_bias=self.dist_bias, sink=self.sink, status=ctx.status, slopes=self.slopes,
                                  q_temp=self.q_temp, gate=gate, chunk=self.chunk or 0)

    # ---- kernels ---------------------------------------------------------------------
    def target_blocks(self) -> int:
        """Decode attention blocks that run at once on this part's device."""
        return DECODE_BLOCKS_PER_SM * ops.sm_count(self.device)

    def uses_flex(self) -> bool:
        """The general form on the tensor cores: bfloat16 and sizes in multiples of 8."""
        return (self.general and self.dtype == torch.bfloat16 and USE_TENSOR_CORES
                and ops.attn_flex_ok(self.H, self.KV, self.hs, self.vs, self.own_v))

    def uses_fast(self, page_size: int) -> bool:
        """The general form whose scores the fast kernels know (the TMA-fed decode kernel, the tcgen05 prompt kernel)."""
        return (self.general and self.plain_scores and self.dtype == torch.bfloat16 and USE_TENSOR_CORES and USE_TMA and USE_TC05
                and max(self.hs, self.vs) <= 128 and self.hs % 8 == 0 and self.vs % 8 == 0 and page_size in (8, 16, 32, 64)
                and self.H // self.KV <= 32 and ops.attn_decode_tma_ok(self.H, self.KV, self.hs, page_size, self.vs)
                and ops.attn_portion_tc05_ok(self.H, self.KV, self.hs, page_size, self.vs))

    def _plan_key(self) -> tuple:
        return ("attention", self.H, self.KV, self.hs, self.vs, self.window, self.chunk)

    def _tag(self) -> str:
        """Names the buffers of a plan: what layers that share it have in common."""
        return f"{self.H}_{self.KV}_{self.hs}_{self.window}" + (f"_v{self.vs}" if self.vs != self.hs else "") \
            + (f"_c{self.chunk}" if self.chunk else "")

    def uses_tensor_cores(self) -> bool:
        return not self.general and self.dtype == torch.bfloat16 and USE_TENSOR_CORES and self.hs % 16 == 0

    def prepare(self, ctx, cache):
        """Cut the step's sequences into work items for the tensor-core kernels: runs of few
        tokens (decode rows) for the decode kernel, longer portions in runs of the portion
        kernel's item size. One plan serves every layer with the same head layout and window."""
        if self.general and not self.uses_fast(cache.page_size):
            if self.uses_flex() and cache.k is not None:
                big = self._plan_general_tc05(ctx, cache.page_size)
                if not big["all"]:
                    flex_plan.plan(ctx, self.device, self.H, self.KV, self.hs, self.vs, self.own_v, self.window, skip=big["skip"],
                                   chunk=self.chunk)
            return
        if not self.general and not self.uses_tensor_cores():
            return
        key = self._plan_key()
        if key in ctx.plans or cache.k is None:
            return
        G = self.H // self.KV
        sizes = (self.H, self.KV, self.hs, cache.page_size) + ((self.vs,) if self.general else ())
        tma = USE_TMA and ops.attn_decode_tma_ok(*sizes)
        dec_rows = ops.attn_decode_tma_rows(self.H, self.KV) if tma else ops.attn_decode_rows(self.H, self.KV, self.hs)
        dec_tokens = dec_rows // G
        tc05 = USE_TC05 and ops.attn_portion_tc05_ok(*sizes)
        por_tokens = (ops.attn_portion_tc05_tokens(self.H, self.KV) if tc05
                      else ops.attn_portion_tokens(self.H, self.KV, self.hs))
        if por_tokens <= 0:
            raise ops.KernelError(f"attention: {G} query heads per kv head do not fit the tensor-core kernels")
        dec, por = [], []
        S = ctx.num_seqs
        qs, cl = ctx.h_q_start, ctx.h_ctx_len
        for s in range(S):
            row0, n = int(qs[s]), int(qs[s + 1] - qs[s])
            pos0 = int(cl[s]) - n
            if n <= dec_tokens:
                dec.append((s, row0, n, pos0))
            else:
                for b in range(0, n, por_tokens):
                    por.append((s, row0 + b, min(por_tokens, n - b), pos0 + b))
        plan = {"dec": None, "por": None, "nsplit": 1, "scratch": None, "tma": tma, "work": None,
                "dec_rows": max((d[2] for d in dec), default=0) * G,
                "tc05": tc05}
        n_dec = len(dec)
        if ctx.seq_cap is not None:                   # fixed shapes: pad with empty items
            dec += [(0, 0, 0, 0)] * (ctx.seq_cap - n_dec)
        if dec and tma:
            # Shares of about equal length for as many blocks as run at once (two per SM), so that a long
            # sequence beside short ones is cut into more of them; a second wave of blocks would wait.
            tiles = []
            for (_, _, n, pos0) in dec:
                first = first_visible_key(pos0, self.window, self.chunk) // 64 * 64
                tiles.append(-(-(pos0 + n - first) // 64) if n > 0 else 0)
            # Entries: every item whole, the shares that run at once, and room for finer cuts when items outnumber
            # those (entries without work are blocks that start and leave, so not more room than pays)
            budget = max(1, self.target_blocks() // self.KV)
            entries = budget + len(dec) + min(3 * len(dec), 2 * budget)
            work = ops.split_work(tiles, budget, entries, MAX_SPLITS, MIN_TILES_PER_SPLIT)
            if ctx.seq_cap is None:                    # shapes are free: only the entries with work
                work = work[:max(1, int((work[:, 0] >= 0).sum()))]
            both = ctx.upload_ints(f"attn_dec_{self._tag()}",
                                   np.concatenate([np.asarray(dec, dtype=np.int32).reshape(-1), work.reshape(-1)]))
            plan["dec"] = both[:4 * len(dec)].view(-1, 4)
            plan["work"] = both[4 * len(dec):].view(-1, 4)
            plan["scratch"] = ctx.buf("attn_split", (ops.attn_decode_tma_work_floats(entries, self.H, self.KV, self.vs),),
                                      torch.float32)
        elif dec:
            # as many blocks as run at once (two per SM), not more: a second wave would wait
            nsplit = max(1, min(MAX_SPLITS, self.target_blocks() // (len(dec) * self.KV)))
            if ctx.seq_cap is None:
                longest = max(d[3] + d[2] for d in dec)
                nsplit = min(nsplit, max(1, -(-longest // (64 * MIN_TILES_PER_SPLIT))))
            plan["nsplit"] = nsplit
            plan["dec"] = ctx.upload_ints(f"attn_dec_{self._tag()}",
                                          np.asarray(dec, dtype=np.int32)).view(-1, 4)
            if nsplit > 1:
                n = ops.attn_decode_scratch_floats(len(dec), self.H, self.KV, self.hs, nsplit)
                plan["scratch"] = ctx.buf("attn_split", (n,), torch.float32)
        if por:
            plan["por"] = ctx.upload_ints(f"attn_por_{self._tag()}",
                                          np.asarray(por, dtype=np.int32)).view(-1, 4)
        ctx.plans[key] = plan

    def attend(self, q, cache, ctx, out):
        if not self.general and not self.uses_tensor_cores():
            ops.paged_attention_ref(q, cache.k, cache.v, cache.block_table, ctx.row_seq, ctx.positions,
                                    out, cache.page_size, ctx.seq_slots, self.H, self.KV, self.hs,
                                    self.scale, self.window or 0, status=ctx.status)
            return
        plan = ctx.plans[self._plan_key()]
        # the fast kernels take chunks and a sink; a layout that has neither may run the others
        extra = {"chunk": self.chunk, "sink": self.sink, "vs": self.vs} if self.general else {}
        args = (cache.page_size, ctx.seq_slots, self.H, self.KV, self.hs, self.scale, self.window or 0)
        if plan["dec"] is not None:
            if plan["tma"]:
                ops.attn_decode_tma(q, cache.k, cache.v, cache.block_table, plan["dec"], out, *args, work=plan["work"],
                                    scratch=plan["scratch"], status=ctx.status, max_rows=plan["dec_rows"], **extra)
            else:
                ops.attn_decode(q, cache.k, cache.v, cache.block_table, plan["dec"], out, *args,
                                nsplit=plan["nsplit"], scratch=plan["scratch"], status=ctx.status)
        if plan["por"] is not None:
            portion = ops.attn_portion_tc05 if plan["tc05"] else ops.attn_portion
            portion(q, cache.k, cache.v, cache.block_table, plan["por"], out, *args, status=ctx.status, **extra)


def distance_bucket(n: int, rows: int, max_distance: float) -> int:
    """Row of a bias table of ``rows`` rows for distance n: its own row below rows/2, then logarithmic steps that
    reach the last row at ``max_distance``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(max_distance / half) * (rows - half))))


def spread_by_distance(table: torch.Tensor, max_distance: float) -> torch.Tensor:
    """fp32 [nd, H] with row n = table[bucket(n)] for every distance up to ``max_distance`` rounded up; distances
    beyond that share the last row, which is what the kernels' ``min(distance, nd - 1)`` gives them."""
    rows = table.shape[0]
    if rows < 2 or max_distance <= rows // 2:
        raise ValueError(f"attention: a bias table of {rows} rows needs max_distance above {rows // 2}, found {max_distance}")
    nd = int(math.ceil(max_distance)) + 1
    idx = torch.tensor([distance_bucket(n, rows, max_distance) for n in range(nd)], dtype=torch.long, device=table.device)
    return table.float().index_select(0, idx).contiguous()


register_mixer("attention", Attention)

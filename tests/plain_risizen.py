"""Plain implementation of the Risizen decoder for the tests: whole sequences, float64, no cache, no batching, one
function per mechanism. It shares no code with the package: it reads config.json and the safetensors file itself and
computes every layer from the equations in each function's docstring.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np
import torch

F64 = torch.float64


# ---- model folder ---------------------------------------------------------------------------

def read_model_folder(folder: str):
    """(config dictionary, {tensor name: float64 or int64 tensor})."""
    with open(os.path.join(folder, "config.json"), "r", encoding="utf-8") as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        data = f.read()
    w = {}
    for name, ent in head.items():
        if name == "__metadata__":
            continue
        a, b = ent["data_offsets"]
        raw = np.frombuffer(data[a:b], dtype=np.uint8)
        dt = ent["dtype"]
        if dt == "BF16":
            u = raw.view("<u2").astype(np.uint32) << 16
            t = torch.from_numpy(u.view(np.float32).astype(np.float64))
        elif dt == "F32":
            t = torch.from_numpy(raw.view("<f4").astype(np.float64))
        elif dt == "I32":
            t = torch.from_numpy(raw.view("<i4").astype(np.int64))
        else:
            raise ValueError(f"dtype {dt} of {name}")
        w[name] = t.reshape(ent["shape"])
    return cfg, w


# ---- mechanisms -----------------------------------------------------------------------------

def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def project(h, w, name):
    """W h + b."""
    return h @ w[name].T + w[name + ".b"]


def short_conv(u, taps):
    """u [T, C], taps [C, K]: y[t, c] = sum_j taps[c, j] u[t - K + 1 + j, c], with u = 0 before the sequence."""
    T, K = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(K):
        back = K - 1 - j
        if back < T:
            y[back:] += taps[:, j] * u[:T - back]
    return y


def chunk_mask(T, size):
    """[T, T] True where query i sees key j: j <= i and both in the same run of ``size`` positions (None: no runs)."""
    i = torch.arange(T).view(-1, 1)
    j = torch.arange(T).view(1, -1)
    m = j <= i
    if size:
        m = m & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))
    return m


def sink_attend(scores, mask, values):
    """scores [H, T, T], values [H, T, dv]: p_j = exp(s_j) / (1 + sum of exp(s)) over the visible keys; sum p_j v_j."""
    s = scores.masked_fill(~mask.unsqueeze(0), -float("inf"))
    top = s.amax(-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(s - top)
    p = e / (torch.exp(-top) + e.sum(-1, keepdim=True))
    return torch.einsum("hij,hjd->ihd", p, values)


def keys_values(h, w, pre, m, eps):
    """k [T, G, dk] = rms(conv(W_k h + b)) per head, v [T, G, dv] = conv(W_v h + b)."""
    T = h.shape[0]
    k = short_conv(project(h, w, pre + "k"), w[pre + "k.conv"]).view(T, m["kv_heads"], m["dim"])
    v = short_conv(project(h, w, pre + "v"), w[pre + "v.conv"]).view(T, m["kv_heads"], m["vdim"])
    return rms(k, eps), v


def attention(h, w, pre, m, eps, kv):
    """q = rms(conv(W_q h + b)) per head; s_h(i, j) = scale q_h(i) . k_g(j), g = h // (H / G), within the chunk; weights with
    one added to the denominator; W_o on the heads side by side. ``kv``: the keys and values to read."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    k, v = kv
    q = rms(short_conv(project(h, w, pre + "q"), w[pre + "q.conv"]).view(T, H, m["dim"]), eps)
    kh = k.repeat_interleave(H // G, dim=1)
    vh = v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kh) * float(m["scale"])
    o = sink_attend(s, chunk_mask(T, (m.get("mask") or {}).get("size")), vh.permute(1, 0, 2))
    return o.reshape(T, -1) @ w[pre + "o"].T


def limited_ff(h, w, pre, limit):
    """g = min(W_gate h, limit); u = clamp(W_up h, -limit, limit); W_down (g sigmoid(1.702 g) (u + 1))."""
    g = torch.clamp(h @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + "up"].T, -limit, limit)
    return (g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)) @ w[pre + "down"].T


def read_streams(x, w, pre):
    """u = sum_s in[s] x_s for x [S, T, d]."""
    return torch.einsum("s,std->td", w[pre + "in"], x)


def write_streams(x, y, w, pre):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, every stream from the old ones."""
    return torch.einsum("sz,std->ztd", w[pre + "mix"], x) + w[pre + "out"].view(-1, 1, 1) * y


# ---- the model --------------------------------------------------------------------------------

def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence. ``layers_out``: a list that receives the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x0 = norm(w["embed"][torch.tensor(list(tokens), dtype=torch.long)], w["embed.norm"], eps)
    x = x0.unsqueeze(0).repeat(int(cfg["streams"]), 1, 1)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(read_streams(x, w, p + "hc1."), w[p + "norm1"], eps)
        src = m.get("kv_from")
        if src is None:
            kept[i] = keys_values(h, w, p + "mix.", m, eps)
        y = attention(h, w, p + "mix.", m, eps, kept[i if src is None else src])
        x = write_streams(x, y, w, p + "hc1.")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(read_streams(x, w, p + "hc2."), w[p + "norm2"], eps)
            x = write_streams(x, limited_ff(h, w, p + "mlp.", float(mlp["limit"])), w, p + "hc2.")
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return norm(x.sum(0), w["final.norm"], eps) @ w["head"].T * float(cfg["logit_scale"])


def greedy(cfg, w, prompt, new):
    """``new`` tokens, each the largest logit after the sequence so far (the whole sequence computed again every time)."""
    toks = list(prompt)
    for _ in range(new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]

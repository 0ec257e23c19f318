"""Plain implementation of the Samulorn decoder for the tests: whole sequences, float64, no cache, no batching,
one function per mechanism. It shares no code with the package: it reads config.json and the safetensors file
itself and computes every layer from the equations in each function's docstring.
"""
from __future__ import annotations

import json
import math
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

def tanh_norm(x, w, name):
    """tanh(alpha x) * weight + bias, entry by entry: no mean, no variance."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def over_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, j] x_{t - (K - 1) + j}, zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    xp = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x], 0)
    return sum(xp[j:j + T] * taps[:, j] for j in range(K))


def delta_head(q, k, v, beta, decay):
    """One head, token by token. q, k [T, dk], v [T, dv], beta [T], decay [T, dk] (a factor per row of S); S is dk x dv:
    S <- diag(decay_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.t() @ q[t])
    return torch.stack(out)


def channel_delta(h, w, p, mx, eps):
    """The mixer 'channel_delta' on normed rows h [T, width]; p: prefix of its tensors."""
    T = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = unit(silu(causal_conv(h @ w[p + "q"].t(), w[p + "q.conv"])).view(T, G, dk)) * dk ** -0.5
    k = unit(silu(causal_conv(h @ w[p + "k"].t(), w[p + "k.conv"])).view(T, G, dk))
    v = silu(causal_conv(h @ w[p + "v"].t(), w[p + "v.conv"])).view(T, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].t())
    low = (h @ w[p + "a1"].t()) @ w[p + "a2"].t()
    step = torch.nn.functional.softplus(low + w[p + "dt_bias"]).view(T, H, dk)
    decay = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * step)
    gate = torch.sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t()).view(T, H, dv)
    heads = []
    for n in range(H):
        g = n // (H // G)
        o = delta_head(q[:, g], k[:, g], v[:, n], beta[:, n], decay[:, n])
        heads.append(over_rms(o, eps) * w[p + "norm"] * gate[:, n])
    return torch.cat(heads, -1) @ w[p + "o"].t()


def frequencies(rot):
    """Angle per position of every pair: base^(-2i/dims), lowered by ``factor`` where the wavelength is long: with
    l = 2 pi / f: f below original/high, f / factor above original/low, and in between the mean of the two with the weight
    s = (original/l - low) / (high - low) on f."""
    f = float(rot["base"]) ** (-2.0 * torch.arange(rot["dims"] // 2, dtype=F64) / rot["dims"])
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for x in f.tolist():
        l = 2.0 * math.pi / x
        if l < sc["original"] / sc["high"]:
            out.append(x)
        elif l > sc["original"] / sc["low"]:
            out.append(x / sc["factor"])
        else:
            s = (sc["original"] / l - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * x / sc["factor"] + s * x)
    return torch.tensor(out, dtype=F64)


def rotate(x, rot):
    """x [T, heads, size]: the neighbouring pairs (2i, 2i + 1) of the first ``dims`` entries are turned by position * f_i."""
    if not rot or rot["dims"] == 0:
        return x
    n = rot["dims"]
    a = torch.arange(x.shape[0], dtype=F64)[:, None, None] * frequencies(rot)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:n:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def causal_attention(q, k, v, scale):
    """One head: softmax over j <= i of scale * q_i . k_j, times v."""
    T = q.shape[0]
    s = (q @ k.t()) * scale
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), -math.inf)
    return torch.softmax(s, -1) @ v


def attention(h, w, p, mx, eps):
    """The left mixer of 'parallel': projections with biases, convolutions, rotation, heads over their root mean square."""
    T = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (causal_conv(h @ w[p + n].t() + w[p + n + ".b"], w[p + n + ".conv"]) for n in ("q", "k", "v"))
    q = over_rms(rotate(q.view(T, H, dk), mx.get("rot")), eps)
    k = over_rms(rotate(k.view(T, G, dk), mx.get("rot")), eps)
    v = v.view(T, G, dv)
    o = [causal_attention(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], mx["scale"]) for n in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].t()


def gated_unit(u, w, p, blocks):
    """The real-gated linear recurrence over u [T, width], token by token:
    r = sigmoid(ra u + b), i = sigmoid(ri u + b) (block-diagonal matrices); a = exp(-8 r softplus(lam));
    S <- a S + sqrt(1 - a^2) i u."""
    T, W = u.shape
    ub = u.view(T, blocks, W // blocks)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w[p + "ra"]) + w[p + "ra.b"]).reshape(T, W)
    i = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w[p + "ri"]) + w[p + "ri.b"]).reshape(T, W)
    la = -8.0 * r * torch.nn.functional.softplus(w[p + "lam"])
    S = torch.zeros(W, dtype=u.dtype)
    out = []
    for t in range(T):
        S = torch.exp(la[t]) * S + torch.sqrt(1.0 - torch.exp(2.0 * la[t])) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def recurrent_block(h, w, p, mx):
    """The right mixer of 'parallel'."""
    y = gelu_tanh(h @ w[p + "y"].t() + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].t() + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    return (gated_unit(u, w, p, mx["blocks"]) * y) @ w[p + "o"].t()


def parallel(h, w, p, mx, eps):
    return (mx["left_scale"] * attention(h, w, p + "left.", mx["left"], eps)
            + mx["right_scale"] * recurrent_block(h, w, p + "right.", mx["right"]))


def gated_feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def choose(s, correction, router):
    """One token's experts: choice scores s + correction; of ``groups.count`` equal runs of neighbours the ``groups.keep`` with
    the largest sum of their two best choice scores stay; the ``top`` best experts among those are chosen."""
    c = s + correction
    E = c.shape[0]
    groups = router.get("groups")
    allowed = torch.ones(E, dtype=torch.bool)
    if groups:
        size = E // groups["count"]
        rank = [(torch.sort(c[g * size:(g + 1) * size], descending=True).values[:2].sum().item(), -g) for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: rank[g], reverse=True)[:groups["keep"]]
        for g in range(groups["count"]):
            if g not in best:
                allowed[g * size:(g + 1) * size] = False
    c = c.masked_fill(~allowed, -math.inf)
    return sorted(range(E), key=lambda e: (-c[e].item(), e))[:router["top"]]


def routed_feed_forward(h, w, p, mlp, margins=None):
    """Every token's chosen experts, weighted by s over the chosen scores' sum (+ 1e-20), times ``scale``. ``margins``: a list
    that gains, per token, how far its choice is from another one (tests leave close calls out)."""
    r = mlp["router"]
    s = torch.sigmoid(h @ w[p + "router"].t())
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(s[t], w[p + "correction"], r)
        if margins is not None:
            margins.append(choice_margin(s[t], w[p + "correction"], r))
        total = sum(s[t, e] for e in ids) + 1e-20
        for e in ids:
            out[t] += r.get("scale", 1.0) * s[t, e] / total * gated_feed_forward(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def choice_margin(s, correction, router):
    """The smallest gap that decides a token's choice: between the last group kept and the first one left out, and between the
    last expert chosen and the first one not chosen among the groups kept."""
    c = s + correction
    E = c.shape[0]
    gaps = []
    groups = router.get("groups")
    allowed = list(range(E))
    if groups and groups["keep"] < groups["count"]:
        size = E // groups["count"]
        rank = [torch.sort(c[g * size:(g + 1) * size], descending=True).values[:2].sum().item() for g in range(groups["count"])]
        order = sorted(range(groups["count"]), key=lambda g: (-rank[g], g))
        gaps.append(rank[order[groups["keep"] - 1]] - rank[order[groups["keep"]]])
        allowed = [e for g in order[:groups["keep"]] for e in range(g * size, (g + 1) * size)]
    best = sorted((c[e].item() for e in allowed), reverse=True)
    if router["top"] < len(best):
        gaps.append(best[router["top"] - 1] - best[router["top"]])
    return min(gaps, default=math.inf)


def token_side_input(x, e, w, p, eps):
    """What a layer adds for the token itself: y = proj (gelu_tanh(gate x) * e), an RMS norm with a weight on y."""
    y = (gelu_tanh(x @ w[p + "gate"].t()) * e) @ w[p + "proj"].t()
    return over_rms(y, eps) * w[p + "norm"]


def run_order(cfg):
    """The layers in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


# ---- the model ------------------------------------------------------------------------------

def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one whole sequence. ``layers_out``: a list that gains the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(list(tokens))
    x = w["embed"][ids] * (cfg.get("embedding") or {}).get("scale", 1.0)
    side = cfg.get("token_side")
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        h = tanh_norm(x, w, p + "norm1")
        if layer["type"] == "channel_delta":
            m = channel_delta(h, w, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "parallel":
            m = parallel(h, w, p + "mix.", layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        x = x + tanh_norm(m, w, p + "norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = tanh_norm(x, w, p + "norm2")
            f = gated_feed_forward(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_feed_forward(h, w, p + "mlp.", mlp, margins)
            x = x + tanh_norm(f, w, p + "norm2b")
        if side:
            d = side["dim"]
            x = x + token_side_input(x, w["side.embed"][ids][:, i * d:(i + 1) * d], w, p + "side.", eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return tanh_norm(x, w, "final.norm") @ w["embed"].t()


def greedy(cfg, w, prompt, n):
    """n greedy tokens after the prompt (each from a forward pass over the whole sequence so far)."""
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(forward(cfg, w, toks)[-1].argmax())
        out.append(nxt)
        toks.append(nxt)
    return out

"""Small Risizen configurations for the tests and a writer of model folders whose weights make every mechanism count: scores
peaked enough that single keys decide, chunks of a few dozen tokens so that every prompt crosses their edges, biases and
convolution taps as large as what they act on, connections between the streams that are far from symmetric, limits that cut a
good part of the gate and up sums. The sizes differ from layer to layer and avoid coincidences (value size != key size, taps
of 1 to 6, one to nine streams, kv_heads == 1 and == heads, layers that read another layer's keys with a longer and with a
shorter chunk, a layer without feed-forward, without chunk, a chunk of one, sizes that are multiples of nothing).
"""
import json
import math
import os

import numpy as np
import torch


def attn(heads, kv, dim, vdim, conv, chunk=None, scale=None, kv_from=None):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale if scale is not None else 3.0 / math.sqrt(dim)}
    if chunk is not None:
        d["mask"] = {"size": chunk}
    if kv_from is not None:
        d["kv_from"] = kv_from
    return d


def dense(ff, limit=1.0):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, streams, eps, layers, logit_scale=1.0):
    return {"architecture": "Risizen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers}


# one mechanism each between embedding and head (a single stream whose connections are plain numbers)
ONLY_ATTN = model(200, 64, 1, 1e-5, [layer(attn(6, 2, 16, 24, 3, chunk=23))], logit_scale=1.7)
# the mixer's output projection is zeroed by the tests that use this one: the feed-forward alone answers
ONLY_DENSE = model(200, 64, 2, 1e-5, [layer(attn(2, 1, 8, 8, 2, chunk=5), dense(72, limit=0.8))])
# keys that other layers read: with a longer chunk, with a shorter one, without any
ONLY_SHARED = model(150, 48, 2, 1e-5, [layer(attn(4, 2, 16, 8, 4, chunk=11)), layer(attn(4, 2, 16, 8, 2, chunk=30, kv_from=0)),
                                       layer(attn(4, 2, 16, 8, 3, chunk=5, kv_from=0)), layer(attn(2, 2, 8, 16, 3, chunk=19)),
                                       layer(attn(2, 2, 8, 16, 1, kv_from=3))])

# all of it, every layer different
MIXED_A = model(331, 96, 3, 1e-5, [
    layer(attn(4, 2, 24, 16, 4, chunk=19), dense(136, limit=0.9)),
    layer(attn(3, 1, 16, 40, 2, chunk=50), dense(72, limit=2.0)),
    layer(attn(4, 2, 24, 16, 3, chunk=33, kv_from=0), None),
    layer(attn(6, 6, 8, 8, 5, chunk=1), dense(96, limit=0.6)),
    layer(attn(3, 1, 16, 40, 4, chunk=13, kv_from=1), dense(40, limit=1.2)),
], logit_scale=0.6)
# sizes that the tensor-core kernels take; key and value heads of 64 and 128 for the TMA-fed kernels
MIXED_B = model(500, 256, 4, 2e-6, [
    layer(attn(4, 2, 64, 64, 4, chunk=72), dense(384, limit=1.1)),
    layer(attn(8, 2, 32, 80, 3, chunk=33), dense(320, limit=0.7)),
    layer(attn(4, 2, 64, 64, 2, chunk=150, kv_from=0), dense(256, limit=1.5)),
    layer(attn(2, 1, 128, 128, 4, chunk=40), None),
    layer(attn(2, 1, 128, 128, 4, kv_from=3), dense(128, limit=1.0)),
], logit_scale=2.5)
# sizes that are multiples of nothing useful, many streams
ODD = model(97, 70, 9, 3e-5, [
    layer(attn(3, 1, 10, 14, 3, chunk=11), dense(50, limit=0.9)),
    layer(attn(5, 5, 6, 10, 6, chunk=27), None),
    layer(attn(3, 1, 10, 14, 2, chunk=64, kv_from=0), dense(18, limit=1.3)),
    layer(attn(6, 3, 7, 5, 1, chunk=6), dense(26, limit=0.5)),
], logit_scale=1.0)
CONFIGS = {"odd": ODD, "attn": ONLY_ATTN, "dense": ONLY_DENSE, "shared": ONLY_SHARED, "mixed_a": MIXED_A, "mixed_b": MIXED_B}
PAGE_SIZE = {"odd": 4, "attn": 8, "dense": 8, "shared": 4, "mixed_a": 8, "mixed_b": 16}


def random_config(rng, aligned):
    """A configuration drawn at random (``rng``: random.Random): two to six layers, chunks from 1 to 300, layers that read
    others' keys, streams, taps, heads, sizes and constants over wide ranges; ``aligned``: sizes in multiples of 8 and key
    sizes that the tensor-core kernels take, else any."""
    m8 = (lambda lo, hi: 8 * rng.randint(max(1, lo // 8), hi // 8)) if aligned else (lambda lo, hi: rng.randint(lo, hi))
    chunks = [1, 2, 5, 16, 17, 31, 48, 64, 100, 300, None]
    layers = []
    for i in range(rng.randint(2, 6)):
        own = [j for j, ly in enumerate(layers) if "kv_from" not in ly["mixer"]]
        if own and rng.random() < 0.4:
            j = rng.choice(own)
            mx = dict(layers[j]["mixer"])
            mx.pop("mask", None)
            mx.update(conv=rng.randint(1, 5), scale=rng.uniform(0.5, 4.0) / math.sqrt(mx["dim"]), kv_from=j)
            c = rng.choice(chunks)
            if c is not None:
                mx["mask"] = {"size": c}
        else:
            kv = rng.choice([1, 2, 3, 4])
            dim = rng.choice([16, 64, 64, 128, 24, 40]) if aligned else rng.randint(4, 72)
            vdim = dim if rng.random() < 0.4 else m8(4, 80)
            mx = attn(kv * rng.choice([1, 2, 3, 4]), kv, dim, vdim, rng.randint(1, 5), chunk=rng.choice(chunks),
                      scale=rng.uniform(0.5, 4.0) / math.sqrt(dim))
        layers.append(layer(mx, None if rng.random() < 0.2 else dense(m8(8, 200), limit=rng.uniform(0.4, 3.0))))
    return model(rng.randint(30, 600), m8(24, 160), rng.choice([1, 2, 2, 3, 4, 4, 5, 8]), rng.choice([1e-6, 1e-5]), layers,
                 logit_scale=rng.uniform(0.3, 3.0))


def silence_mixer(t):
    """For the configuration that tests a feed-forward alone: the mixer's output projection becomes zero."""
    t["l0.mix.o"][:] = 0.0


def _tensors(cfg, seed):
    """{name: float32 array}, from a numpy generator; rounded to bfloat16 when written."""
    rng = np.random.default_rng(seed)
    W, S = cfg["width"], cfg["streams"]
    out = {}

    def lin(name, n_out, n_in, gain=1.0):
        out[name] = (rng.standard_normal((n_out, n_in)) * gain / math.sqrt(n_in)).astype(np.float32)

    def vec(name, n, mean=0.0, std=1.0):
        out[name] = (mean + std * rng.standard_normal(n)).astype(np.float32)

    def connections(p):
        vec(p + "in", S, 0.7, 0.4)
        vec(p + "out", S, 1.0, 0.4)
        out[p + "mix"] = (0.75 * np.eye(S) + 0.35 / math.sqrt(S) * rng.standard_normal((S, S))).astype(np.float32)

    out["embed"] = rng.standard_normal((cfg["vocab"], W)).astype(np.float32) * 2.0
    vec("embed.norm", W, 1.0, 0.2)
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = ly["mixer"]
        q = p + "mix."
        H, G, dk, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        vec(p + "norm1", W, 1.0, 0.15)
        connections(p + "hc1.")
        for name, rows in [("q", H * dk)] + ([] if "kv_from" in m else [("k", G * dk), ("v", G * dv)]):
            lin(q + name, rows, W)
            vec(q + name + ".b", rows, 0.0, 0.4)
            taps = 0.45 * rng.standard_normal((rows, K))
            taps[:, -1] += 0.9
            out[q + name + ".conv"] = taps.astype(np.float32)
        lin(q + "o", W, H * dv)
        mlp = ly.get("mlp")
        if mlp is None:
            continue
        vec(p + "norm2", W, 1.0, 0.15)
        connections(p + "hc2.")
        f = p + "mlp."
        lin(f + "gate", mlp["ff"], W, 1.5); lin(f + "up", mlp["ff"], W, 1.5); lin(f + "down", W, mlp["ff"])
    vec("final.norm", W, 1.0, 0.1)
    lin("head", cfg["vocab"], W, 3.0)
    return out


def write_folder(folder, cfg, seed, change=None):
    """A model folder with the weights above in bfloat16. ``change(tensors)`` may edit the float32 arrays first (a test
    that builds a key which stands out, say)."""
    from llm_steadyinfer_b200.weights import write_safetensors
    os.makedirs(folder, exist_ok=True)
    arrays = _tensors(cfg, seed)
    if change is not None:
        change(arrays)
    tensors = {n: torch.tensor(a).to(torch.bfloat16) for n, a in arrays.items()}
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f, indent=1)
    return folder

"""Small Samulorn configurations for the tests and a writer of model folders whose weights make every mechanism count: scores
peaked enough that single keys decide, decays near enough to one that old tokens are still read, biases and convolution taps as
large as what they act on, norms that bend (tanh of arguments around one), corrections that move experts and groups past one another.
The sizes differ from layer to layer and avoid coincidences (value size != key size, taps of 1 to 6, kv_heads == 1 and == heads, parts
of any size, ranks that are no multiple of 8, groups that are all kept and groups of one, a layer without feed-forward, without
rotation, with a part of a head rotated, scales that differ, loops in the middle, sizes that are multiples of nothing).
"""
import json
import math
import os

import numpy as np
import torch


def delta(heads, kv, dim, vdim, conv, rank=12):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "rank": rank}


def rot(dims, base=900.0, scaling=(4.0, 1.0, 4.0, 60)):
    d = {"base": base, "dims": dims}
    if scaling is not None:
        d["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return d


def pair(left, right, ls=1.0, rs=1.0):
    """left: (heads, kv, dim, vdim, conv, rot or None); right: (width, blocks, conv)"""
    h, kv, dim, vdim, conv, r = left
    a = {"heads": h, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": 2.5 / math.sqrt(dim)}
    if r is not None:
        a["rot"] = r
    return {"left": a, "right": dict(zip(("width", "blocks", "conv"), right)), "left_scale": ls, "right_scale": rs}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, scale=1.0):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "channel_delta", "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, side=None, loop=None, eps=1e-5, scale=2.0):
    d = {"architecture": "Samulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if side is not None:
        d["token_side"] = {"dim": side}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# one mechanism each between embedding and head
ONLY_DELTA = model(200, 64, [layer(delta(4, 2, 24, 16, 4))])
ONLY_PAIR = model(200, 64, [layer(pair((6, 2, 16, 24, 3, rot(16)), (48, 3, 2), 1.3, 0.7))])
# the mixers of these say nothing (their second norm is zeroed): the feed-forward, or the token input, answers alone
ONLY_MOE = model(200, 64, [layer(delta(2, 1, 8, 8, 2), moe(24, 12, 3, (4, 2), 1.7))])
ONLY_DENSE = model(200, 64, [layer(delta(2, 1, 8, 8, 2), dense(72))])
ONLY_SIDE = model(200, 64, [layer(delta(2, 1, 8, 8, 2)), layer(delta(2, 1, 8, 8, 2))], side=20)
ONLY_LOOP = model(150, 48, [layer(delta(2, 2, 16, 8, 3)), layer(pair((4, 4, 8, 16, 2, rot(4, scaling=None)), (32, 2, 3)))], loop=(0, 2, 3))

# all of it, every layer different
MIXED_A = model(331, 96, [
    layer(delta(6, 2, 24, 16, 3, rank=10), dense(136)),
    layer(pair((4, 2, 24, 16, 4, rot(24)), (72, 3, 4), 0.8, 1.4), moe(40, 10, 3, (5, 3), 2.5)),
    layer(delta(4, 4, 16, 40, 5, rank=20), None),
    layer(pair((3, 1, 16, 8, 1, rot(8, base=50.0)), (40, 5, 3), 1.2, 0.6), moe(24, 6, 2, None, 1.0)),
    layer(delta(3, 1, 40, 24, 2), moe(16, 9, 4, (3, 3), 0.7)),
], side=12, loop=(1, 3, 2))
# sizes that the tensor-core kernels take; key and value heads of 64 and 128 for the TMA-fed kernels
MIXED_B = model(500, 256, [
    layer(pair((4, 2, 64, 64, 3, rot(64, base=10000.0, scaling=(8.0, 1.0, 4.0, 128))), (256, 4, 4), 1.1, 0.9), moe(64, 16, 4, (4, 2), 2.0)),
    layer(delta(4, 2, 64, 64, 4, rank=24), dense(320)),
    layer(pair((2, 1, 128, 128, 4, rot(64, scaling=None)), (128, 8, 2), 0.5, 1.5), None),
    layer(delta(2, 2, 128, 128, 2, rank=64), moe(96, 8, 2, (8, 4), 1.5)),
], side=32, loop=(1, 4, 2), eps=2e-6, scale=16.0)
# sizes that are multiples of nothing useful
ODD = model(97, 70, [
    layer(delta(6, 3, 10, 14, 3, rank=7), moe(18, 7, 2, None, 1.3)),
    layer(pair((3, 1, 10, 14, 6, rot(6)), (30, 6, 5), 0.9, 1.1), dense(50)),
    layer(pair((5, 5, 14, 10, 2, None), (33, 1, 1), 1.0, 1.0), None),
    layer(delta(2, 1, 13, 9, 6, rank=3), moe(10, 15, 5, (5, 2), 0.9)),
    layer(delta(3, 1, 11, 15, 1, rank=1), dense(26)),
], side=5, eps=3e-5, loop=(3, 5, 1))
CONFIGS = {"odd": ODD, "delta": ONLY_DELTA, "pair": ONLY_PAIR, "moe": ONLY_MOE, "dense": ONLY_DENSE, "side": ONLY_SIDE, "loop": ONLY_LOOP,
           "mixed_a": MIXED_A, "mixed_b": MIXED_B}
PAGE_SIZE = {"odd": 4, "delta": 8, "pair": 8, "moe": 16, "dense": 4, "side": 8, "loop": 4, "mixed_a": 8, "mixed_b": 16}


def random_config(rng, aligned):
    """A configuration drawn at random (``rng``: random.Random): one to five layers of both kinds, all sizes and constants over wide
    ranges; ``aligned``: sizes in multiples of 8 and key sizes that the tensor-core kernels take, else any."""
    m8 = (lambda lo, hi: 8 * rng.randint(max(1, lo // 8), hi // 8)) if aligned else (lambda lo, hi: rng.randint(lo, hi))
    layers = []
    for _ in range(rng.randint(1, 5)):
        kv = rng.choice([1, 2, 3, 4])
        dim = rng.choice([16, 64, 64, 128, 24, 40]) if aligned else rng.randint(10, 72)
        vdim = dim if rng.random() < 0.4 else m8(10, 80)
        if rng.random() < 0.5:
            mx = delta(kv * rng.choice([1, 2, 3]), kv, dim, vdim, rng.randint(1, 5), rank=rng.randint(1, 40))
        else:
            dims = rng.choice([0, dim // 2 // 2 * 2, dim // 2 * 2])
            r = None if rng.random() < 0.15 else rot(dims, rng.choice([100.0, 10000.0, 500000.0]),
                                                     None if rng.random() < 0.3 else (rng.uniform(1.5, 8.0), 1.0, rng.uniform(2.0, 5.0), rng.choice([40, 150, 2048])))
            blocks = rng.choice([1, 2, 3, 4, 6])
            mx = pair((kv * rng.choice([1, 2, 3, 4]), kv, dim, vdim, rng.randint(1, 5), r), (blocks * m8(4, 40), blocks, rng.randint(1, 5)),
                      rng.uniform(0.3, 1.6), rng.uniform(0.3, 1.6))
        kind = rng.random()
        if kind < 0.2:
            mlp = None
        elif kind < 0.5:
            mlp = dense(m8(8, 200))
        else:
            size, count = rng.randint(1, 4), rng.randint(2, 5)
            keep = rng.randint(1, count)
            mlp = moe(m8(8, 64), size * count, rng.randint(1, min(4, keep * size)), (count, keep) if rng.random() < 0.8 else None, rng.uniform(0.5, 3.0))
        layers.append(layer(mx, mlp))
    loop = None
    if rng.random() < 0.6:
        a = rng.randrange(len(layers))
        loop = (a, rng.randint(a + 1, len(layers)), rng.randint(1, 3))
    return model(rng.randint(30, 600), m8(24, 160), layers, side=None if rng.random() < 0.2 else rng.randint(1, 40), loop=loop,
                 eps=rng.choice([1e-6, 1e-5]), scale=rng.uniform(0.5, 10.0))


def silence_mixers(t):
    """For the configurations that test a feed-forward or the token input alone: what the mixer says becomes zero."""
    for n in t:
        if n.endswith(".norm1b") or n.endswith(".norm1b.b"):
            t[n][:] = 0.0


CHANGES = {"moe": silence_mixers, "dense": silence_mixers, "side": silence_mixers}


def _tensors(cfg, seed):
    """{name: float32 array}, from a numpy generator; rounded to bfloat16 when written."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    out = {}

    def lin(name, n_out, n_in, gain=1.0):
        out[name] = (rng.standard_normal((n_out, n_in)) * gain / math.sqrt(n_in)).astype(np.float32)

    def vec(name, n, mean=0.0, std=1.0):
        out[name] = (mean + std * rng.standard_normal(n)).astype(np.float32)

    def norm(name, alpha=0.6):
        vec(name, W, 1.0, 0.2)
        vec(name + ".b", W, 0.0, 0.2)
        out[name + ".alpha"] = np.array(alpha * rng.uniform(0.7, 1.4), np.float32)

    def conv(name, channels, K):
        taps = 0.45 * rng.standard_normal((channels, K))
        taps[:, -1] += 0.9
        out[name] = taps.astype(np.float32)

    vec("embed", (cfg["vocab"], W), 0.0, 1.5 / cfg["embedding"]["scale"])
    side = cfg.get("token_side")
    if side:
        vec("side.embed", (cfg["vocab"], len(cfg["layers"]) * side["dim"]))
    for i, ly in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", ly["mixer"]
        q = p + "mix."
        norm(p + "norm1"); norm(p + "norm1b", 0.9)
        if ly["type"] == "channel_delta":
            H, G, dk, dv, K, r = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["conv"], mx["rank"]
            for n, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                lin(q + n, c, W, 1.3); conv(q + n + ".conv", c, K)
            lin(q + "b", H, W, 1.5)
            out[q + "A_log"] = np.log(rng.uniform(0.3, 4.0, H)).astype(np.float32)
            lin(q + "a1", r, W); lin(q + "a2", H * dk, r)
            out[q + "dt_bias"] = rng.uniform(-6.0, -1.0, H * dk).astype(np.float32)     # decays of 0.9 to 0.999 a token
            lin(q + "g1", r, W, 1.5); lin(q + "g2", H * dv, r, 1.5)
            vec(q + "norm", dv, 1.0, 0.2)
            lin(q + "o", W, H * dv, 2.0)
        else:
            left, right = mx["left"], mx["right"]
            H, G, dk, dv, K = left["heads"], left["kv_heads"], left["dim"], left["vdim"], left["conv"]
            for n, c in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                lin(q + "left." + n, c, W, 1.3); vec(q + f"left.{n}.b", c, 0.0, 0.4); conv(q + f"left.{n}.conv", c, K)
            lin(q + "left.o", W, H * dv, 1.5)
            R, B, K = right["width"], right["blocks"], right["conv"]
            q += "right."
            lin(q + "y", R, W, 1.5); vec(q + "y.b", R, 0.5, 0.5)
            lin(q + "x", R, W, 1.3); vec(q + "x.b", R, 0.0, 0.4)
            conv(q + "conv", R, K); vec(q + "conv.b", R, 0.0, 0.3)
            for n in ("ra", "ri"):
                out[q + n] = (rng.standard_normal((B, R // B, R // B)) * 1.5 / math.sqrt(R // B)).astype(np.float32)
                vec(q + n + ".b", (B, R // B), 0.0, 0.6)
            out[q + "lam"] = rng.uniform(-7.0, -2.0, R).astype(np.float32)              # decays of 0.4 to 0.996 at r = 1
            lin(q + "o", W, R, 1.5)
        mlp = ly.get("mlp")
        if mlp is not None:
            norm(p + "norm2"); norm(p + "norm2b", 0.9)
            f = p + "mlp."
            if mlp["kind"] == "dense":
                F = mlp["ff"]
                lin(f + "gate", F, W, 1.7); lin(f + "up", F, W, 1.7); lin(f + "down", W, F, 1.7)
            else:
                F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
                for n, rows, cols in (("gate", F, W), ("up", F, W), ("down", W, F)):
                    # experts that resemble one another: a choice that rounding turns must not drown everything behind it
                    lin("common", rows, cols, 1.6)
                    common = out.pop("common")
                    for e in range(E):
                        lin(f"{f}e{e}.{n}", rows, cols, 0.35)
                        out[f"{f}e{e}.{n}"] += common
                lin(f + "router", E, W, 2.5)
                vec(f + "correction", E, -0.3, 0.35)         # choice scores of both signs
        if side:
            D = side["dim"]
            lin(p + "side.gate", D, W); lin(p + "side.proj", W, D); vec(p + "side.norm", W, 0.5, 0.2)
    norm("final.norm", 0.5)
    vec("final.norm", W, 0.0, 1.0)                       # of both signs: the head is the embedding, and a token must not simply echo itself
    return out


def write_folder(folder, cfg, seed, change=None):
    """A model folder with the weights above in bfloat16. ``change(tensors)`` may edit the float32 arrays first (a test that builds a key
    which stands out, say)."""
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

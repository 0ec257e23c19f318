"""Risizen on the GPU against the plain implementation (tests/plain_risizen.py): every mechanism alone, prompts against
token-by-token decoding, portions down to two tokens, unequal batches with pages and slots used again, keys just inside and
just outside every chunk and at page borders, layers that read another layer's keys, the first tokens, long decoding, other
sizes, and greedy generation through the entry point. Weights come from tests/risizen_configs.py, which makes them so that a
lost key, a chunk that is one token off, a forgotten bias, tap, sink or stream shows in the logits."""
import json
import math
import os
import random
import subprocess
import sys

import pytest
import torch

import plain_risizen as pr
import replay_util as ru
import risizen_configs as rc

pytestmark = pytest.mark.gpu

# A row's error: root mean square of the difference of the logits (mean taken off) over that of the plain logits. In 32-bit
# every row is held to the limit. In bfloat16 rounding alone gives a median well below it with single rows above: the limit
# holds for the median and for all but one row in twenty, and no row may pass four times the limit.
LIMIT = {torch.float32: 2e-4, torch.bfloat16: 8e-2}
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]
DEV = "cuda:0"
CHANGES = {"dense": rc.silence_mixer}


class Plain(ru.PlainLogits):
    def __init__(self, folder):
        super().__init__(folder, pr)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("risizen")
    return {n: rc.write_folder(os.path.join(str(root), n), cfg, seed=71 + i, change=CHANGES.get(n))
            for i, (n, cfg) in enumerate(rc.CONFIGS.items())}


@pytest.fixture(scope="module")
def plains(folders):
    return {n: Plain(d) for n, d in folders.items()}


def replayer(folder, name, dtype, max_tokens, max_requests=4):
    from llm_steadyinfer_b200.engine.replay import Replayer
    return Replayer(folder, dtype, max_tokens, page_size=rc.PAGE_SIZE[name], max_requests=max_requests)


def row_error(row, ref):
    d = row.to(torch.float64) - ref
    d = d - d.mean()
    return (d.pow(2).mean().sqrt() / ref.sub(ref.mean()).pow(2).mean().sqrt()).item()


def check(rp, steps, reqs, plain, dtype, what):
    worst, n, errors = 0.0, 0, []
    hard = LIMIT[dtype] * (4 if dtype == torch.bfloat16 else 1)
    for rid, p, row in ru.replay_in_process(rp, steps):
        assert torch.isfinite(row).all(), f"{what}: request {rid!r} position {p}: logits are not finite"
        e = row_error(row, plain.of(reqs[rid])[p])
        assert e == e and e <= hard, f"{what}: request {rid!r} position {p}: error {e:.3e} (allowed {hard:.0e})"
        worst, n = max(worst, e), n + 1
        errors.append(e)
    assert n > 0
    if dtype == torch.bfloat16:
        errors.sort()
        over = sum(e > LIMIT[dtype] for e in errors)
        assert over <= max(1, n // 20), f"{what}: {over} of {n} rows above {LIMIT[dtype]:.0e}"
        assert errors[n // 2] <= LIMIT[dtype] / 2 or n < 4, f"{what}: median error {errors[n // 2]:.3e}"
    mgr = rp.runner.manager
    mgr.check_invariant()
    assert not mgr.requests
    assert all(mgr.free_pages(g) == mgr.groups[g].pool.num_pages for g in range(len(mgr.groups)))
    return worst


def requests_of(name, lengths, seed=0):
    vocab = rc.CONFIGS[name]["vocab"]
    return {f"q{i}": ru.random_tokens(vocab, n, 1000 * seed + i) for i, n in enumerate(lengths)}


# ---- each mechanism alone, and the layers of a whole model one by one ------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["attn", "dense", "shared"])
def test_each_mechanism_alone(folders, plains, name, dtype):
    """A one-layer model of the mixer without feed-forward, one of the feed-forward beside a mixer whose output projection is
    zero, and one of layers that read others' keys: the logits whole and token by token."""
    reqs = requests_of(name, [1, 2, 37, 90])
    for mode, steps in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail(reqs, tail=30))):
        check(replayer(folders[name], name, dtype, 128), steps, reqs, plains[name], dtype, f"{name}/{mode}")


@pytest.mark.parametrize("name", ["mixed_a", "mixed_b", "odd", "shared"])
def test_layers_one_by_one_in_32_bit(folders, name):
    """The sum of the streams after every layer against the plain one."""
    toks = ru.random_tokens(rc.CONFIGS[name]["vocab"], 75, 5)
    cfg, w = pr.read_model_folder(folders[name])
    want = []
    pr.forward(cfg, w, toks, layers_out=want)
    rp = replayer(folders[name], name, torch.float32, 128)
    got = {}
    rp.runner.model.hook_layers(lambda run, x: got.__setitem__(run, x.double().cpu()))
    rp.run_step([{"id": "a", "tokens": toks, "want": [len(toks) - 1]}], end=["a"])
    assert sorted(got) == list(range(len(cfg["layers"])))
    for run in range(len(cfg["layers"])):
        scale = want[run].abs().max().item()
        diff = (got[run] - want[run]).abs().max().item()
        assert diff <= 5e-5 * scale, f"{name}: layer {run} differs by {diff:.2e} of {scale:.1f}"


# ---- schedules ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["mixed_a", "mixed_b", "odd"])
@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "mixed"])
def test_schedules(folders, plains, name, dtype, mode):
    reqs = requests_of(name, [1, 3, 19, 64, 65, 130, 201], seed=1)
    longest = ru.round64(max(len(t) for t in reqs.values()))
    if mode == "whole":
        steps, max_tokens = ru.trace_whole(reqs), longest
    elif mode == "tail":
        steps, max_tokens = ru.trace_tail(reqs, tail=40), longest
    elif mode == "portions":
        steps, max_tokens = ru.trace_portions(reqs, sizes=(2, 17, 3, 2, 31, 5, 64, 2, 9, 1, 40)), longest
    else:
        max_tokens = longest + 128                       # two or three live at a time: pages and slots come again
        steps = ru.trace_mixed(reqs, max_tokens, seed=3, max_live=3)
    rp = replayer(folders[name], name, dtype, max_tokens, max_requests=3)
    worst = check(rp, steps, reqs, plains[name], dtype, f"{name}/{mode}")
    print(f"{name} {mode} {dtype}: worst row error {worst:.2e}")


def test_prompt_equals_token_by_token_in_32_bit(folders):
    """The same request whole, one token a step, and in portions of two: the logits agree far below the distance to the
    plain implementation (the kernels differ between the three, the function does not)."""
    name = "mixed_a"
    toks = ru.random_tokens(rc.CONFIGS[name]["vocab"], 70, 12)
    reqs = {"a": toks}
    runs = []
    for steps in (ru.trace_whole(reqs), ru.trace_portions(reqs, sizes=(1,)), ru.trace_portions(reqs, sizes=(2,))):
        rp = replayer(folders[name], name, torch.float32, 128)
        runs.append(torch.stack([row for _, _, row in ru.replay_in_process(rp, steps)]).double())
    for other in runs[1:]:
        e = max(row_error(other[i], runs[0][i]) for i in range(len(toks)))
        assert e < 2e-5, f"prompt and steps differ by {e:.2e}"


def test_a_long_portion_beside_short_ones_and_single_tokens(folders, plains):
    """One step holds a portion long enough for the prompt kernels of many rows, a short portion and single tokens of
    requests that are further on: each sequence takes its own kernel, and every row its own past and chunk."""
    name = "mixed_b"
    reqs = requests_of(name, [300, 40, 170, 9], seed=6)
    t = reqs
    steps = [
        {"step": 0, "entries": [{"id": "q0", "tokens": t["q0"][:140], "want": [0, 139]}, {"id": "q1", "tokens": t["q1"][:39], "want": [38]}], "end": []},
        {"step": 1, "entries": [{"id": "q0", "tokens": t["q0"][140:299], "want": [0, 1, 2, 4, 70, 158]}, {"id": "q1", "tokens": t["q1"][39:], "want": [0]},
                                {"id": "q2", "tokens": t["q2"][:5], "want": [4]}, {"id": "q3", "tokens": t["q3"][:2], "want": [0, 1]}], "end": ["q1"]},
        {"step": 2, "entries": [{"id": "q2", "tokens": t["q2"][5:169], "want": list(range(0, 164, 13))}, {"id": "q0", "tokens": t["q0"][299:], "want": [0]},
                                {"id": "q3", "tokens": t["q3"][2:], "want": [0, 6]}], "end": ["q0", "q3"]},
        {"step": 3, "entries": [{"id": "q2", "tokens": t["q2"][169:], "want": [0]}], "end": ["q2"]},
    ]
    for dtype in DTYPES:
        check(replayer(folders[name], name, dtype, 640), steps, reqs, plains[name], dtype, "long beside short")


def test_batch_equals_alone_and_slots_come_again(folders, plains):
    """Unequal requests in one batch against each alone, with two request slots for five requests: every slot and page is
    used again, and the keys and convolution inputs that the request before left there must not show."""
    name, dtype = "mixed_a", torch.float32
    reqs = requests_of(name, [70, 9, 33, 2, 51], seed=2)
    rp = replayer(folders[name], name, dtype, 192, max_requests=2)
    check(rp, ru.trace_mixed(reqs, 192, seed=9, max_live=2, prompt_frac=0.5), reqs, plains[name], dtype, "two slots")
    again = dict(reversed(list(reqs.items())))
    check(rp, ru.trace_mixed(again, 192, seed=10, max_live=2, prompt_frac=0.3), again, plains[name], dtype, "two slots again")


def test_requests_cut_back_and_computed_again(folders, plains):
    """Preemption in a trace: with chunks and convolution inputs nothing of a cut request can be kept, and what is computed
    again equals the first time."""
    name = "mixed_a"
    reqs = requests_of(name, [70, 33, 90], seed=8)
    rp = replayer(folders[name], name, torch.float32, 256, max_requests=3)
    steps = ru.trace_mixed(reqs, 256, seed=5, max_live=3, cut_every=4, kept=rp.kept_after_truncate)
    assert any("truncate" in s for s in steps)
    check(rp, steps, reqs, plains[name], torch.float32, "cut back")


@pytest.mark.parametrize("name", ["mixed_a", "mixed_b"])
def test_long_decoding(folders, plains, name):
    """A short prompt, then 300 tokens one by one: every chunk begins and ends among decoded tokens, and pages that no layer
    reads any more go back to the pool."""
    reqs = requests_of(name, [310], seed=3)
    for dtype in DTYPES:
        check(replayer(folders[name], name, dtype, 320), ru.trace_tail(reqs, tail=300), reqs, plains[name], dtype, "long decoding")


def test_first_tokens(folders, plains):
    """Positions 0, 1, 2 alone and as the start of portions: a convolution whose past is not there yet, a softmax over one
    key and the sink."""
    for name in ("mixed_b", "odd"):
        reqs = requests_of(name, [1, 2, 3, 5], seed=4)
        for dtype in DTYPES:
            for sizes in ((1,), (2, 1), (1, 2)):
                check(replayer(folders[name], name, dtype, 64), ru.trace_portions(reqs, sizes=sizes), reqs, plains[name], dtype, f"first tokens {sizes}")


@pytest.mark.parametrize("dim,vdim,page", [(16, 24, 8), (64, 64, 16), (12, 10, 4)])
def test_a_key_at_the_chunk_edge_decides(tmp_path, dim, vdim, page):
    """One layer, one tap, one stream: the logits of a chunk's last row depend on the token at the chunk's start and not on
    the one before it, in the plain implementation; the engine must follow in prompts, in portions cut at the edge and in
    single tokens."""
    chunk = 21
    cfg = rc.model(120, 64, 1, 1e-5, [rc.layer(rc.attn(4, 2, dim, vdim, 1, chunk=chunk))])
    folder = rc.write_folder(str(tmp_path / "edge"), cfg, 6)
    plain = Plain(folder)
    n = 4 * chunk
    a = ru.random_tokens(120, n, 78)
    inside, outside = list(a), list(a)
    shows = lambda t: row_error(pr.forward(plain.cfg, plain.w, a[:n - chunk] + [t] + a[n - chunk + 1:])[-1], plain.of(a)[-1])
    inside[n - chunk] = max(range(0, 120, 3), key=shows)          # the last row still sees this place (a token that stands out there)
    outside[n - chunk - 1] = inside[n - chunk]                    # and not this one
    assert row_error(plain.of(inside)[-1], plain.of(a)[-1]) > 50 * LIMIT[torch.float32], "the key inside the chunk does not count"
    assert row_error(plain.of(outside)[-1], plain.of(a)[-1]) < 1e-9, "the key outside the chunk counts"
    rc.PAGE_SIZE["edge"] = page
    for dtype in DTYPES:
        reqs = {"a": a, "in": inside, "out": outside}
        check(replayer(folder, "edge", dtype, 128), ru.trace_portions(reqs, sizes=(n - chunk - 1, 1, 2, chunk - 3, 1)), reqs, plain, dtype, "chunk edge, portions")
        check(replayer(folder, "edge", dtype, 128), ru.trace_tail(reqs, tail=chunk + 5), reqs, plain, dtype, "chunk edge, decoding")


def test_other_sizes_where_the_usual_ones_coincide(tmp_path):
    """Sizes that a model may make equal or one: a single head, one stream, one tap, a chunk of one and of two, no chunk,
    no feed-forward anywhere but at the end."""
    cfg = rc.model(64, 32, 1, 1e-5, [
        rc.layer(rc.attn(1, 1, 12, 12, 1, chunk=1)),
        rc.layer(rc.attn(2, 1, 8, 4, 2, chunk=2)),
        rc.layer(rc.attn(2, 2, 4, 16, 17)),
        rc.layer(rc.attn(2, 2, 4, 16, 1, chunk=200, kv_from=2), rc.dense(8, limit=0.3)),
    ], logit_scale=5.0)
    folder = rc.write_folder(str(tmp_path / "small"), cfg, 8)
    plain = Plain(folder)
    reqs = {f"q{i}": ru.random_tokens(64, n, 50 + i) for i, n in enumerate([1, 2, 7, 40])}
    for dtype in DTYPES:
        check(replayer(folder, "odd", dtype, 64), ru.trace_portions(reqs, sizes=(3, 2, 1, 9)), reqs, plain, dtype, "small sizes")


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Layer orders, readers of other layers' keys, head counts, sizes, chunks, taps, streams and constants drawn at random
    (even seeds: sizes that the tensor-core kernels take): every schedule in 32-bit, whole prompts and a mixed batch in
    bfloat16."""
    rng = random.Random(500 + seed)
    cfg = rc.random_config(rng, aligned=seed % 2 == 0)
    rc.PAGE_SIZE["random"] = 16 if seed % 2 == 0 else rng.choice([4, 8, 16])
    folder = rc.write_folder(str(tmp_path / "m"), cfg, 500 + seed)
    plain = Plain(folder)
    lens = [1, 2, rng.randint(3, 40), rng.randint(60, 130), rng.randint(150, 300)]
    reqs = {f"q{i}": ru.random_tokens(cfg["vocab"], n, 7 * seed + i) for i, n in enumerate(lens)}
    longest = ru.round64(max(lens))
    for dtype, modes in ((torch.float32, ("whole", "tail", "portions", "mixed")), (torch.bfloat16, ("whole", "mixed"))):
        for mode in modes:
            if mode == "whole":
                steps, mt = ru.trace_whole(reqs), longest
            elif mode == "tail":
                steps, mt = ru.trace_tail(reqs, tail=40), longest
            elif mode == "portions":
                steps, mt = ru.trace_portions(reqs, sizes=(2, 17, 3, 2, 31, 5, 64, 2, 9, 1, 40, 100)), longest
            else:
                mt = longest + 128
                steps = ru.trace_mixed(reqs, mt, seed=seed, max_live=4)
            check(replayer(folder, "random", dtype, mt, max_requests=4), steps, reqs, plain, dtype, f"random {seed}/{mode}")


# ---- kernels ----------------------------------------------------------------------------------------------

def _paged(rows, page_size, perm_seed):
    """rows [n, heads, d] into a shuffled page pool; returns (cache [pages, heads, page_size, d], table [1, blocks])."""
    n, KV, d = rows.shape
    blocks = -(-n // page_size)
    g = torch.Generator().manual_seed(perm_seed)
    pages = torch.randperm(blocks + 3, generator=g)[:blocks]
    cache = torch.zeros(blocks + 3, KV, page_size, d, dtype=rows.dtype)
    for j in range(n):
        cache[pages[j // page_size], :, j % page_size] = rows[j]
    return cache, pages.to(torch.int32).view(1, -1)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,G,dk,dv,chunk,sink", [(4, 2, 24, 16, 37, 0.0), (8, 2, 48, 72, 100, 0.0), (3, 1, 10, 6, 64, 1.5), (6, 6, 16, 8, 1, 0.0),
                                                  (4, 2, 64, 64, 50, 0.0), (8, 2, 128, 128, 129, 0.0), (4, 1, 128, 128, None, 6.0),
                                                  (16, 1, 64, 64, 96, 0.0), (2, 2, 64, 64, 16, 0.7), (24, 1, 64, 64, 70, 0.0),
                                                  (4, 2, 104, 64, 60, 0.0), (6, 2, 56, 120, 45, 0.0), (4, 4, 8, 8, 20, 0.0)])
def test_attention_with_chunks_and_sink(H, G, dk, dv, chunk, sink, dtype):
    """Queries built so that one key would carry nearly all of a head's weight: the last key before the row's chunk (must
    not count), the chunk's first key from its last rows, keys at page borders, the row's own key; the other rows' scores are
    small, so that the sink takes a good part of their weight. Rows run as a prompt and once more one by one, through every
    kernel that takes the sizes: the plain one, mma.sync (keys whole and in shares), the TMA-fed decode kernel, tcgen05."""
    from llm_steadyinfer_b200.csrc import ops
    torch.manual_seed(3 + H)
    n, ps, last = 330, 16, 70
    ratio = H // G
    c = chunk or n
    k = torch.randn(n, G, dk) * 0.3
    q = torch.randn(n, H, dk) * 0.3
    v = torch.randn(n, G, dv)
    edge = (n - 1) // c * c                                       # start of the last row's chunk
    wanted = [(edge, edge - 1), (edge + 1, edge), (n - 1, edge), (n - 2, edge - 1), (n - 3, (n - 3) // ps * ps), (n - 4, (n - 4) // ps * ps - 1),
              (n - 5, n - 5), (n - 6, 0), (min(n - 7, edge + 2), edge + 1), (edge - 1, max(0, edge - c))]
    taken = set()
    for i, j in wanted:
        if 0 <= j <= i < n and i not in taken and j >= 0:
            taken.add(i)
            k[j] = k[j] / k[j].norm(dim=-1, keepdim=True) * 6.0
            for h in range(H):
                q[i, h] = k[j, h // ratio] * (1.5 if h % 2 else 1.0)
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    scale = 0.5
    kh, vh = k.repeat_interleave(ratio, dim=1), v.repeat_interleave(ratio, dim=1).permute(1, 0, 2)
    s = torch.einsum("ihd,jhd->hij", q, kh) * scale

    def result(size, sk):
        # exp(sk) in the denominator: the plain form with every score taken relative to sk
        return pr.sink_attend(s - sk, pr.chunk_mask(n, size), vh).reshape(n, H * dv)

    want = result(chunk, sink)
    if chunk and edge - 1 >= 0:
        seen = pr.chunk_mask(n, None)
        other = pr.sink_attend(s - sink, seen, vh).reshape(n, H * dv)
        assert (other[edge] - want[edge]).abs().max() > 0.05, "the key before the chunk would not show"
    assert (result(chunk, -50.0)[n - last:] - want[n - last:]).abs().max() > 0.05, "the sink would not show"
    qd = q.reshape(n, H * dk).to(dtype).to(DEV)
    kc, table = _paged(k.to(dtype), ps, 3)
    vc, _ = _paged(v.to(dtype), ps, 3)
    kc, vc, table = kc.to(DEV), vc.to(DEV), table.to(DEV)
    seqs, posd = torch.zeros(n, dtype=torch.int32, device=DEV), torch.arange(n, dtype=torch.int32, device=DEV)
    sd = torch.full((H,), sink, dtype=torch.float32, device=DEV)
    limit = 1e-4 if dtype == torch.float32 else 4e-2
    cd = chunk or 0

    def compare(out, ref, what):
        diff = (out.double().cpu() - ref).abs().max().item()
        assert diff <= limit, f"{what}: differs by {diff:.2e}"

    out = torch.zeros(n, H * dv, dtype=dtype, device=DEV)
    ops.attention_general(qd, kc, vc, table, seqs, posd, out, ps, 1, H, G, dk, dv, scale, sink=sd, chunk=cd)
    compare(out, want, "plain kernel")
    if dtype != torch.bfloat16 or not ops.attn_flex_ok(H, G, dk, dv, True):
        return
    per = ops.attn_flex_tokens(H, G)
    items = torch.tensor([(0, b, min(per, n - b), b) for b in range(0, n, per)], dtype=torch.int32, device=DEV)
    out.zero_()
    ops.attn_flex(qd, kc, vc, table, items, out, ps, 1, H, G, dk, dv, scale, sink=sd, chunk=cd)
    compare(out, want, "mma.sync, prompt rows")
    singles = lambda: torch.tensor([(0, r, 1, n - last + r) for r in range(last)], dtype=torch.int32, device=DEV)
    for nsplit in (1, 3):
        one = torch.zeros(last, H * dv, dtype=dtype, device=DEV)
        scratch = torch.zeros(ops.attn_flex_scratch_floats(last, H, G, dv, nsplit), dtype=torch.float32, device=DEV) if nsplit > 1 else None
        ops.attn_flex(qd[n - last:], kc, vc, table, singles(), one, ps, 1, H, G, dk, dv, scale, sink=sd, chunk=cd, nsplit=nsplit,
                      scratch=scratch, max_rows=ratio)
        compare(one, want[n - last:], f"mma.sync, single rows in {nsplit} shares")
    if ops.attn_portion_tc05_ok(H, G, dk, ps, dv):
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        per = ops.attn_portion_tc05_tokens(H, G)
        items = torch.tensor([(0, b, min(per, n - b), b) for b in range(0, n, per)], dtype=torch.int32, device=DEV)
        out.zero_()
        ops.attn_portion_tc05(qd, kc, vc, table, items, out, ps, 1, H, G, dk, scale, status=status, chunk=cd, sink=sd, vs=dv)
        assert status.item() == 0
        compare(out, want, "tcgen05, prompt rows")
        if ops.attn_decode_tma_ok(H, G, dk, ps, dv):
            for nsplit in (1, 3):
                one = torch.zeros(last, H * dv, dtype=dtype, device=DEV)
                scratch = torch.zeros(max(1, ops.attn_decode_tma_scratch_floats(last, H, G, dv, nsplit)), dtype=torch.float32, device=DEV)
                ops.attn_decode_tma(qd[n - last:], kc, vc, table, singles(), one, ps, 1, H, G, dk, scale, nsplit=nsplit, scratch=scratch,
                                    status=status, max_rows=ratio, chunk=cd, sink=sd, vs=dv)
                compare(one, want[n - last:], f"TMA decode, single rows in {nsplit} shares")
            few = ops.attn_decode_tma_rows(H, G) // ratio          # items of several tokens, some over a chunk's edge
            items = torch.tensor([(0, b, min(few, last - b), n - last + b) for b in range(0, last, few)], dtype=torch.int32, device=DEV)
            one = torch.zeros(last, H * dv, dtype=dtype, device=DEV)
            ops.attn_decode_tma(qd[n - last:], kc, vc, table, items, one, ps, 1, H, G, dk, scale, status=status, chunk=cd, sink=sd, vs=dv)
            compare(one, want[n - last:], "TMA decode, several rows an item")
            assert status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("NQ,NK,NV,dk,dv,K,norm,bias", [(6, 2, 2, 16, 24, 4, True, True), (4, 4, 4, 64, 64, 4, True, True), (5, 0, 0, 48, 8, 3, True, True),
                                                        (8, 2, 2, 128, 40, 2, True, False), (2, 1, 1, 8, 8, 1, True, True), (3, 1, 1, 10, 6, 3, True, True),
                                                        (2, 2, 2, 32, 16, 7, True, True), (2, 1, 1, 256, 128, 4, False, True), (1, 1, 1, 264, 72, 4, True, True)])
@pytest.mark.parametrize("times", [1, 24], ids=["few_rows", "many_rows"])
def test_convolution_norm_and_store(NQ, NK, NV, dk, dv, K, norm, bias, times, dtype):
    """The launch behind the stacked projection: three sequences cut into portions of changing size (single rows, two rows,
    portions shorter and longer than the taps, all in unequal batches, a padding row behind them), the state carried in slots
    that held something else before, keys and values found in their pages; and with portions many times as long, whose rows
    several blocks share."""
    from llm_steadyinfer_b200.csrc import ops
    torch.manual_seed(K + dk)
    C = (NQ + NK) * dk + NV * dv
    lens, ps, slots, eps = [41 * times, 23 * times, 60 * times], 8, [3, 0, 2], 1e-5
    pad = -(-C // 8) * 8 + 8                                       # rows with further columns behind
    u = {s: torch.randn(n, pad).to(dtype) for s, n in enumerate(lens)}
    taps = (torch.randn(K, C) * 0.6).to(torch.bfloat16).float()
    b = (torch.randn(C) * 0.4).to(torch.bfloat16).float() if bias else None
    want = {}
    for s in u:
        p = u[s][:, :C].double() + (b.double() if bias else 0.0)
        y = pr.short_conv(p, taps.double().T)
        n = lens[s]
        q, k, v = y[:, :NQ * dk].view(n, NQ, dk), y[:, NQ * dk:(NQ + NK) * dk].view(n, NK, dk), y[:, (NQ + NK) * dk:].view(n, NV, dv)
        want[s] = (pr.rms(q, eps), pr.rms(k, eps), v) if norm else (q, k, v)
    stride = -(-(K - 1) * C // 4) * 4
    state = torch.full((4, stride), 7.0, device=DEV) if K > 1 else None
    blocks = -(-max(lens) // ps)
    pages = torch.randperm(3 * blocks + 2, generator=torch.Generator().manual_seed(1))[:3 * blocks].view(3, blocks)
    table = pages.to(torch.int32).to(DEV)
    kc = torch.zeros(3 * blocks + 2, max(NK, 1), ps, dk, dtype=dtype, device=DEV)
    vc = torch.zeros(3 * blocks + 2, max(NV, 1), ps, dv, dtype=dtype, device=DEV)
    got_q = {s: torch.zeros(n, NQ * dk, dtype=dtype) for s, n in enumerate(lens)}
    at = [0, 0, 0]
    sizes = [(1, 2, 17), (1, 1, 1), (2, 3, 1), (1, 5, 2), (20, 0, 9), (3, 1, 30), (0, 11, 0), (13, 0, 0)]
    sizes = [tuple(m * times if m > 1 else m for m in step) for step in sizes] + [(times, times, times)] * 3
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    for step in sizes:
        live = [(s, min(m, lens[s] - at[s])) for s, m in enumerate(step) if min(m, lens[s] - at[s]) > 0]
        if not live:
            continue
        rows = torch.cat([u[s][at[s]:at[s] + m] for s, m in live] + [torch.full((1, pad), 9.0).to(dtype)]).to(DEV)
        pos = [p for s, m in live for p in range(at[s], at[s] + m)] + [0]
        seq = [i for i, (_, m) in enumerate(live) for _ in range(m)] + [-1]
        starts = [0]
        for _, m in live:
            starts.append(starts[-1] + m)
        q = torch.zeros(len(pos), NQ * dk, dtype=dtype, device=DEV)
        portions = (1 if any(m > 1 and at[s] == 0 for s, m in live) else 0) | (2 if any(m > 1 and at[s] > 0 for s, m in live) else 0)
        ops.qkv_conv(rows, b.to(DEV) if bias else None, taps.to(DEV), state, i32(pos), i32(seq), i32(starts), i32([at[s] + m for s, m in live]),
                     i32([slots[s] for s, _ in live]), table[[s for s, _ in live]].contiguous(), kc if NK else None, vc if NK else None, ps, len(live),
                     NQ, NK, NV, dk, dv, q, norm, eps, portions=portions, status=status)
        r = 0
        for s, m in live:
            got_q[s][at[s]:at[s] + m] = q[r:r + m].cpu()
            r += m
            at[s] += m
    assert at == lens and status.item() == 0
    tol = 2e-5 if dtype == torch.float32 else 5e-3
    off = lambda got, ref: ((got.double() - ref).abs() / (1.0 + ref.abs())).max().item()
    for s, n in enumerate(lens):
        assert off(got_q[s].view(n, NQ, dk), want[s][0]) < tol, f"queries of sequence {s}"
        if NK:
            at_page, place = pages[s, torch.arange(n) // ps], torch.arange(n) % ps
            assert off(kc.cpu()[at_page, :, place], want[s][1]) < tol, f"keys of sequence {s}"
            assert off(vc.cpu()[at_page, :, place], want[s][2]) < tol, f"values of sequence {s}"
        if K > 1:                                                  # the slot holds the last taps - 1 projected values
            kept = state[slots[s], :(K - 1) * C].cpu().double().view(K - 1, C)
            assert (kept - (u[s][n - K + 1:, :C].double() + (b.double() if bias else 0.0))).abs().max() < 1e-6
    if K > 1:
        assert (state[1] == 7.0).all()                             # a slot that no sequence holds


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("T,S,d", [(1, 4, 4096), (3, 2, 256), (17, 3, 1000), (300, 4, 2048), (5, 1, 64), (9, 5, 96), (4, 8, 520), (6, 9, 70), (2, 2, 33),
                                   (700, 2, 136), (2, 3, 20000), (3, 2, 2052), (2, 7, 4100), (40, 4, 2048)])
def test_streams_written_read_and_normalised(T, S, d, dtype):
    """x' = mix^T x + write y, u = read . x', the norm of u: in place, from one row that stands for all streams, without a
    result to write (the first sublayer), for chosen rows and the plain sum (the end of the model)."""
    from llm_steadyinfer_b200.csrc import ops
    torch.manual_seed(T + S)
    x = torch.randn(T, S, d)
    x0 = torch.randn(T, d)
    y = torch.randn(T, d).to(dtype)
    w = {"p.in": torch.randn(S), "p.out": torch.randn(S), "p.mix": torch.randn(S, S)}
    wd = {n: t.to(DEV) for n, t in w.items()}
    w = {n: t.double() for n, t in w.items()}
    w2 = {"p.in": torch.randn(S, dtype=torch.float64)}
    weight = 1.0 + 0.2 * torch.randn(d)
    weight = weight.to(torch.bfloat16) if T % 2 else weight         # both storage types of a norm's weight
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    eps = 1e-5
    run = lambda src, out, **kw: ops.stream_norm(src, weight.to(DEV), eps, out, streams=S, **kw)
    close = lambda got, ref, t: (got.double().cpu() - ref).abs().max().item() <= t * max(1.0, ref.abs().max().item())
    conn = dict(y=y.to(DEV), mix=wd["p.mix"], write=wd["p.out"], read=w2["p.in"].float().to(DEV))

    def plain(streams):                                            # [T, S, d] -> streams after, the norm of what is read
        new = pr.write_streams(streams.double().permute(1, 0, 2), y.double(), w, "p.")
        u = pr.read_streams(new, w2, "p.")
        return new.permute(1, 0, 2), u

    new, u = plain(x)
    src = x.to(DEV).clone()
    out = torch.zeros(T, d, dtype=dtype, device=DEV)
    run(src, out, dst=src, **conn)
    assert close(src, new, 1e-5) and close(out, pr.norm(u, weight.double(), eps), tol)
    # chosen rows, the sum of the streams, nothing stored
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device=DEV)
    picked = torch.zeros(3, d, dtype=dtype, device=DEV)
    keep = x.to(DEV).clone()
    run(keep, picked, rows=rows, y=conn["y"], mix=conn["mix"], write=conn["write"])
    assert torch.equal(keep.cpu(), x)
    assert close(picked, pr.norm(new.sum(1), weight.double(), eps)[rows.cpu().long()], tol)
    # one row for all streams: before the first result, then the first result written
    run(x0.to(DEV), out, read=conn["read"])
    assert close(out, pr.norm(x0.double() * w2["p.in"].sum(), weight.double(), eps), tol)
    new, u = plain(x0.unsqueeze(1).expand(T, S, d))
    dst = torch.full((T, S, d), 9.0, device=DEV)
    ahead = torch.zeros(1 << 16, dtype=torch.bfloat16, device=DEV)
    run(x0.to(DEV), out, dst=dst, ahead=ahead, **conn)
    assert close(dst, new, 1e-5) and close(out, pr.norm(u, weight.double(), eps), tol)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d", [64, 70, 2048])
def test_embedding_with_a_norm(d, dtype):
    from llm_steadyinfer_b200.csrc import ops
    torch.manual_seed(d)
    table = torch.randn(50, d).to(dtype)
    w = 1.0 + 0.2 * torch.randn(d)
    toks = torch.tensor([3, 49, 0, 3, 7], dtype=torch.int32)
    out = torch.zeros(5, d, device=DEV)
    ops.embedding_gather(toks.to(DEV), table.to(DEV), out, scale=1.5, norm_weight=w.to(DEV), eps=1e-5)
    want = pr.norm(1.5 * table[toks.long()].double(), w.double(), 1e-5)
    assert (out.double().cpu() - want).abs().max() < 1e-5


# ---- the entry point ----------------------------------------------------------------------------------------

def greedy(cfg, w, prompt, new):
    """``new`` greedy tokens of the plain implementation, and the smallest gap between the two best logits on the way."""
    toks, gap = list(prompt), math.inf
    for _ in range(new):
        logits = pr.forward(cfg, w, toks)[-1]
        top2 = torch.topk(logits, 2).values
        gap = min(gap, (top2[0] - top2[1]).item())
        toks.append(int(logits.argmax()))
    return toks[len(prompt):], gap


@pytest.mark.parametrize("name", ["mixed_a", "mixed_b"])
def test_greedy_generation_through_the_entry_point(folders, name):
    """Greedy tokens through LLM (scheduler, sampler, graphs and steps launched ahead) equal the plain implementation's
    in 32-bit; bfloat16 runs and mostly agrees."""
    from llm_steadyinfer_b200 import LLM, SamplingParams
    cfg, w = pr.read_model_folder(folders[name])
    prompts = [ru.random_tokens(cfg["vocab"], n, 50 + n) for n in (5, 23, 1, 40)]
    both = [greedy(cfg, w, p, 12) for p in prompts]
    want = [b[0] for b in both]
    assert min(b[1] for b in both) > 1e-3, "the test's prompts meet a close call between two tokens"
    for dtype in ("float32", "bfloat16"):
        for graphs in (True, False):
            llm = LLM(folders[name], dtype=dtype, max_batch=3, max_seq_len=64, max_gen_len=12, block_size=rc.PAGE_SIZE[name],
                      max_num_batched_tokens=32, use_cuda_graph=graphs, async_decode=graphs)
            got = [g.token_ids for g in llm.generate(prompts, SamplingParams(ignore_eos=True))]
            if dtype == "float32":
                assert got == want, f"{name} graphs={graphs}: {got} != {want}"
            else:
                same = sum(a == b for g, x in zip(got, want) for a, b in zip(g, x))
                assert same >= 24, f"{name} bf16: only {same} of 48 tokens agree"
            if graphs:
                assert llm.runner.graphs_available() and llm.stats["graph_steps"] > 0


def test_preemption_recomputes_from_the_start(folders):
    """A pool too small for all requests: some are cut back and computed again, and the tokens still equal the plain
    implementation's."""
    from llm_steadyinfer_b200 import LLM, SamplingParams
    name = "mixed_a"
    cfg, w = pr.read_model_folder(folders[name])
    prompts = [ru.random_tokens(cfg["vocab"], n, 90 + n) for n in (30, 28, 26)]
    want = [greedy(cfg, w, p, 20)[0] for p in prompts]
    llm = LLM(folders[name], dtype="float32", max_batch=3, max_seq_len=64, max_gen_len=20, block_size=8, num_blocks=14,
              max_num_batched_tokens=64)
    assert [r.token_ids for r in llm.generate(prompts, SamplingParams(ignore_eos=True))] == want


def test_trace_program_replays_a_mixed_trace(folders, plains, tmp_path):
    """``bin/trace_run`` as a program: a mixed trace in 32-bit, its files and its "done" lines."""
    name = "mixed_a"
    reqs = requests_of(name, [40, 3, 90, 17, 66], seed=7)
    steps = ru.trace_mixed(reqs, 256, seed=1, max_live=3)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders[name], "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "256", "--page-size", str(rc.PAGE_SIZE[name])],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    pos, vocab = {}, rc.CONFIGS[name]["vocab"]
    for rec in steps:
        wanted = sum(len(e["want"]) for e in rec["entries"])
        rows = None
        if wanted:
            rows = torch.from_file(str(out / f"{rec['step']}.f32"), size=wanted * vocab, dtype=torch.float32).view(wanted, vocab)
        r = 0
        for e in rec["entries"]:
            base = pos.get(e["id"], 0)
            for wpos in e["want"]:
                assert row_error(rows[r], plains[name].of(reqs[e["id"]])[base + wpos]) <= LIMIT[torch.float32]
                r += 1
            pos[e["id"]] = base + len(e["tokens"])


def test_command_line_serves_the_design(folders, tmp_path):
    """The serving program on a Risizen folder: requests of random lengths arriving over time, sampling, a pool that is
    used again; and once more on random weights drawn from a configuration file."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "m.json"
    common = ["--num-requests", "12", "--max-batch", "4", "--max-gen", "10", "--prompt-len-dist", "lognormal:30,0.7,2,90",
              "--output-len-dist", "lognormal:6,0.5,1,10", "--request-rate", "300", "--temperature", "0.8", "--top-p", "0.9",
              "--ignore-eos", "--kv-block-size", "8", "--num-kv-blocks", "60", "--max-num-batched-tokens", "40",
              "--max-model-len", "128", "--output-json", str(out)]
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(rc.MIXED_A))
    for source in (["--checkpoint", folders["mixed_a"]], ["--model-config", str(cfg_file)]):
        proc = subprocess.run([sys.executable, os.path.join(root, "bin", "offline_batch_benchmark"), *source, *common],
                              capture_output=True, text=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-3000:]
        m = json.loads(out.read_text())[0]
        assert m["completed"] == 12 and m["rejected"] == 0 and m["output_tokens"] > 12 and m["output_tps"] > 0

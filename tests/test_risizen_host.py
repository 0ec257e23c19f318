"""Risizen without a GPU: configuration (keys, errors, round trip), the model as a specification (streams, attention with
biases, convolutions, chunks and a sink, layers that read another layer's keys), checkpoint names and shapes, cache and state
places, how long the cache keeps keys that several layers read, what the parts make of their weights, and the plain
implementation's own consistency (closed forms of its mechanisms)."""
import copy
import math
import random

import pytest
import torch

import plain_risizen as pr
import risizen_configs as rc
from llm_steadyinfer_b200.cache import CacheLayout, CacheManager
from llm_steadyinfer_b200.config import ConfigError, config_from_dict, load_config
from llm_steadyinfer_b200.models import Model
from llm_steadyinfer_b200.parts import CacheNeed
from llm_steadyinfer_b200.weights.loader import load_weights_into

F64 = torch.float64


def test_configuration_round_trip_and_spec():
    cfg = config_from_dict(rc.MIXED_A)
    assert config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    assert spec.order == [0, 1, 2, 3, 4] and spec.vocab_size == 331 and spec.hidden_size == 96 and spec.streams == 3
    assert spec.logit_scale == 0.6 and spec.embedder.params["norm"] == {"eps": 1e-5, "name": "embed.norm"}
    assert all(l.arrangement == "streams" and l.mixer_streams_prefix == "hc1." for l in spec.layers)
    assert [l.feed_forward_streams_prefix for l in spec.layers] == ["hc2.", "hc2.", None, "hc2.", "hc2."]
    assert [l.cache_from for l in spec.layers] == [None, None, 0, None, 1]
    a = spec.layers[0].mixer
    assert a.kind == "attention" and a.position is None and a.params["chunk"] == 19 and a.params["conv_taps"] == 4
    assert a.params["biases"] and a.params["qk_norm"] == {"eps": 1e-5} and a.params["sink_score"] == 0.0 and a.params["own_keys"]
    b = spec.layers[2].mixer
    assert not b.params["own_keys"] and b.params["chunk"] == 33 and b.params["conv_taps"] == 3
    ff = spec.layers[0].feed_forward
    assert ff.kind == "gated_mlp_limited" and ff.params["limit"] == 0.9 and ff.params["alpha"] == 1.702 and not ff.params["biases"]
    assert config_from_dict(rc.ONLY_SHARED).model_spec().layers[4].mixer.params["chunk"] is None


@pytest.mark.parametrize("edit,word", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d.pop("streams"), "streams"),
    (lambda d: d.update(streams=0), "streams"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.update(logit_scale="big"), "logit_scale"),
    (lambda d: d.update(layers=[]), "layers"),
    (lambda d: d["layers"][0].update(type="mamba"), "type"),
    (lambda d: d["layers"][0].pop("mixer"), "mixer"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda d: d["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
    (lambda d: d["layers"][2]["mixer"].update(kv_from=1), "layer 1"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
])
def test_configuration_errors_name_the_key(edit, word):
    d = copy.deepcopy(rc.MIXED_A)
    edit(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


def test_checkpoint_names_shapes_cache_and_state_places(tmp_path):
    folder = rc.write_folder(str(tmp_path / "m"), rc.MIXED_A, 3)
    model = Model(load_config(folder), torch.float32, "cpu")
    shapes = model.weight_shapes()
    assert shapes["embed"] == (331, 96) and shapes["embed.norm"] == (96,) and shapes["head"] == (331, 96) and shapes["final.norm"] == (96,)
    assert shapes["l0.hc1.in"] == (3,) and shapes["l0.hc1.out"] == (3,) and shapes["l0.hc2.mix"] == (3, 3) and "l2.hc2.mix" not in shapes
    assert shapes["l0.mix.q"] == (96, 96) and shapes["l0.mix.q.b"] == (96,) and shapes["l0.mix.q.conv"] == (96, 4)
    assert shapes["l0.mix.v"] == (32, 96) and shapes["l0.mix.v.conv"] == (32, 4) and shapes["l0.mix.o"] == (96, 64)
    assert "l2.mix.k" not in shapes and "l2.mix.v.conv" not in shapes and "l2.mix.k.b" not in shapes and shapes["l2.mix.q.conv"] == (96, 3)
    assert set(shapes) == set(rc._tensors(rc.MIXED_A, 0))
    load_weights_into(model, folder)
    needs, states = model.cache_places()
    assert len(needs) == 6 and needs[-1] is None and states[-1] is None
    assert (needs[0].num_kv_heads, needs[0].head_dim, needs[0].v_dim, needs[0].chunk, needs[0].window) == (2, 24, 16, 19, None)
    assert needs[2].layout_key() == needs[0].layout_key() and needs[2].chunk == 33
    # the convolutions' last taps - 1 values: of q, k and v, or of q alone where the keys are another layer's
    assert states[0].shape == (3 * (96 + 48 + 32),) and states[2].shape == (2 * 96,) and states[3].shape == (4 * 144,)
    assert model.capturable()


def test_state_of_one_tap_and_odd_sizes(tmp_path):
    folder = rc.write_folder(str(tmp_path / "m"), rc.ODD, 3)
    model = Model(load_config(folder), torch.float32, "cpu")
    _, states = model.cache_places()
    assert states[3] is None                                       # one tap: nothing to remember
    assert states[0].shape == (2 * (30 + 10 + 14),) and states[1].shape == (-(-5 * (30 + 30 + 50) // 4) * 4,)


def test_what_the_parts_make_of_their_weights(tmp_path):
    folder = rc.write_folder(str(tmp_path / "m"), rc.MIXED_A, 4)
    model = Model(load_config(folder), torch.float32, "cpu")
    load_weights_into(model, folder)
    _, w = pr.read_model_folder(folder)
    b = model.blocks[0]
    assert torch.equal(b.mixer_streams.mix.double(), w["l0.hc1.mix"]) and torch.equal(b.feed_forward_streams.read.double(), w["l0.hc2.in"])
    a = b.mixer
    assert torch.equal(a.qkv.double(), torch.cat([w["l0.mix.q"], w["l0.mix.k"], w["l0.mix.v"]]))
    assert torch.equal(a.qkv_bias.double(), torch.cat([w["l0.mix.q.b"], w["l0.mix.k.b"], w["l0.mix.v.b"]]))
    assert torch.equal(a.qkv_taps.double(), torch.cat([w["l0.mix.q.conv"], w["l0.mix.k.conv"], w["l0.mix.v.conv"]]).T)
    assert a.sink.tolist() == [0.0] * 4
    r = model.blocks[2].mixer
    assert torch.equal(r.qkv.double(), w["l2.mix.q"]) and r.qkv_taps.shape == (3, 96) and r.channels == 96
    # the logits' scale sits in the final norm's weight
    assert torch.allclose(model.final_norm.weight.double(), w["final.norm"] * 0.6, rtol=1e-6)
    assert torch.equal(model.embedder.norm_weight.double(), w["embed.norm"])


def test_random_weights_draw_connections_around_the_identity():
    from llm_steadyinfer_b200.weights.random_init import random_tensors
    model = Model(config_from_dict(rc.ONLY_SHARED), torch.float32, "cpu")
    t = random_tensors(model, 0, torch.float32)
    assert (t["l0.hc1.mix"] - torch.eye(2)).abs().max() < 0.13 and (t["l0.hc1.mix"] - torch.eye(2)).abs().max() > 0
    assert (t["l0.hc1.in"] - 1).abs().max() < 0.7 and t["l0.mix.q.conv"].abs().max() < 0.13


# ---- the cache under chunks and several readers ------------------------------------------------------------

def _manager(needs, cache_from=None, page_size=4, num_pages=64):
    return CacheManager(CacheLayout(needs, [None] * len(needs), cache_from), page_size, num_pages, 4)


def test_chunks_give_pages_back_at_their_edge():
    m = _manager([CacheNeed(1, 8, chunk=10), CacheNeed(1, 8, chunk=10), CacheNeed(1, 8)])
    assert len(m.groups) == 2 and m.groups[0].layers == [0, 1]
    m.admit("a")
    length = 0
    for n in (3, 6, 1, 1, 12, 1, 1, 1, 1, 1, 9, 40):
        m.grow("a", length + n)
        length += n
        m.commit("a", length)
        start = length // 10 * 10                        # the next token's chunk begins here
        for b, p in enumerate(m.table(0, "a")):
            assert (p < 0) == ((b + 1) * 4 <= start), (length, b)
        assert all(p >= 0 for p in m.table(1, "a"))
        m.check_invariant()
    assert m.can_truncate_to(20) == 0
    m.release("a")
    assert m.free_pages(0) == 64 and m.free_pages(1) == 64


def test_pages_are_kept_for_the_reader_that_looks_back_furthest():
    need = lambda chunk=None, window=None: CacheNeed(1, 8, window=window, chunk=chunk)
    lay = CacheLayout([need(6), need(6), need(20), need(window=9)], [None] * 4, [None, None, 1, 1])
    assert lay.num_groups == 2 and lay.layer_group == [0, 1, 1, 1]
    m = CacheManager(lay, 4, 64, 4)
    m.admit("a")
    for length in range(1, 90):
        m.grow("a", length)
        m.commit("a", length)
        alone, shared = length // 6 * 6, min(length // 6 * 6, length // 20 * 20, max(0, length - 8))
        assert [p < 0 for p in m.table(0, "a")] == [(b + 1) * 4 <= alone for b in range(len(m.table(0, "a")))]
        assert [p < 0 for p in m.table(1, "a")] == [(b + 1) * 4 <= shared for b in range(len(m.table(1, "a")))]
        m.check_invariant()
    # a reader without limits keeps everything
    m = _manager([need(6), need()], [None, 0])
    m.admit("a"); m.grow("a", 50); m.commit("a", 50)
    assert not m.groups[0].bounded and all(p >= 0 for p in m.table(0, "a"))


def test_chunked_requests_at_random_keep_the_invariant():
    rng = random.Random(4)
    m = _manager([CacheNeed(2, 8, chunk=7), CacheNeed(2, 8, chunk=18), CacheNeed(1, 8, chunk=3)], [None, 0, None], num_pages=40)
    live, nxt = {}, 0
    for _ in range(500):
        if rng.random() < 0.2 and len(live) < 4:
            m.admit(nxt); live[nxt] = 0; nxt += 1
        elif live and rng.random() < 0.85:
            r = rng.choice(list(live))
            n = rng.randint(1, 9)
            if m.can_grow(r, live[r] + n):
                m.grow(r, live[r] + n); live[r] += n; m.commit(r, live[r])
        elif live:
            r = rng.choice(list(live))
            m.release(r); del live[r]
        m.check_invariant()


# ---- the plain implementation ---------------------------------------------------------------------------------

def test_plain_convolution():
    u = torch.tensor([[1.0, 2.0], [3.0, 5.0], [7.0, 11.0], [13.0, 17.0]], dtype=F64)
    taps = torch.tensor([[100.0, 10.0, 1.0], [0.0, 1.0, 0.0]], dtype=F64)
    y = pr.short_conv(u, taps)
    assert y[:, 0].tolist() == [1.0, 13.0, 137.0, 383.0]           # the last tap is the current token's
    assert y[:, 1].tolist() == [0.0, 2.0, 5.0, 11.0]
    assert torch.equal(pr.short_conv(u[:1], taps), y[:1])


def test_plain_chunks_and_sink():
    m = pr.chunk_mask(7, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1] and m[5].tolist() == [False, False, False, True, True, True, False]
    assert pr.chunk_mask(4, None).sum().item() == 10
    s = torch.tensor([[[0.3, 0.0], [-1.0, 2.0]]], dtype=F64)
    v = torch.tensor([[[1.0], [10.0]]], dtype=F64)
    out = pr.sink_attend(s, pr.chunk_mask(2, None), v)
    e = math.exp
    assert abs(out[0, 0, 0].item() - e(0.3) / (1 + e(0.3))) < 1e-12
    assert abs(out[1, 0, 0].item() - (e(-1.0) + 10 * e(2.0)) / (1 + e(-1.0) + e(2.0))) < 1e-12
    # scores far below the sink's leave nothing, far above it everything
    assert pr.sink_attend(s - 900.0, pr.chunk_mask(2, None), v).abs().max() == 0.0
    assert torch.allclose(pr.sink_attend(s + 900.0, pr.chunk_mask(2, 1), v)[:, 0, 0], v[0, :, 0])


def test_plain_streams():
    torch.manual_seed(0)
    S, T, d = 3, 4, 5
    x, y = torch.randn(S, T, d, dtype=F64), torch.randn(T, d, dtype=F64)
    w = {"p.in": torch.randn(S, dtype=F64), "p.out": torch.randn(S, dtype=F64), "p.mix": torch.randn(S, S, dtype=F64)}
    new = pr.write_streams(x, y, w, "p.")
    for t in range(S):
        assert torch.allclose(new[t], sum(w["p.mix"][s, t] * x[s] for s in range(S)) + w["p.out"][t] * y)
    assert torch.allclose(pr.read_streams(x, w, "p."), sum(w["p.in"][s] * x[s] for s in range(S)))
    # plain connections are the usual residual sum
    one = {"p.in": torch.ones(1, dtype=F64), "p.out": torch.ones(1, dtype=F64), "p.mix": torch.ones(1, 1, dtype=F64)}
    assert torch.allclose(pr.write_streams(x[:1], y, one, "p.")[0], x[0] + y) and torch.equal(pr.read_streams(x[:1], one, "p."), x[0])


def test_plain_model_puts_the_pieces_in_order():
    cfg = rc.model(20, 8, 2, 1e-5, [rc.layer(rc.attn(2, 1, 4, 6, 2, chunk=3), rc.dense(6, limit=0.7)),
                                    rc.layer(rc.attn(2, 1, 4, 6, 3, chunk=2, kv_from=0), None)], logit_scale=1.3)
    w = {n: torch.tensor(a, dtype=F64) for n, a in rc._tensors(cfg, 1).items()}
    toks = [3, 7, 7, 1, 19, 0]
    layers = []
    logits = pr.forward(cfg, w, toks, layers_out=layers)
    eps = 1e-5
    x0 = pr.norm(w["embed"][toks], w["embed.norm"], eps)
    x = torch.stack([x0, x0])
    m0, m1 = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    h = pr.norm(w["l0.hc1.in"].sum() * x0, w["l0.norm1"], eps)
    kv = pr.keys_values(h, w, "l0.mix.", m0, eps)
    x = pr.write_streams(x, pr.attention(h, w, "l0.mix.", m0, eps, kv), w, "l0.hc1.")
    h = pr.norm(pr.read_streams(x, w, "l0.hc2."), w["l0.norm2"], eps)
    g, u = torch.clamp(h @ w["l0.mlp.gate"].T, max=0.7), torch.clamp(h @ w["l0.mlp.up"].T, -0.7, 0.7)
    assert (h @ w["l0.mlp.gate"].T > 0.7).any() and (h @ w["l0.mlp.up"].T < -0.7).any()
    x = pr.write_streams(x, (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w["l0.mlp.down"].T, w, "l0.hc2.")
    assert torch.allclose(layers[0], x.sum(0))
    h = pr.norm(pr.read_streams(x, w, "l1.hc1."), w["l1.norm1"], eps)
    x = pr.write_streams(x, pr.attention(h, w, "l1.mix.", m1, eps, kv), w, "l1.hc1.")       # the first layer's keys, its own chunk
    assert torch.allclose(layers[1], x.sum(0))
    assert torch.allclose(logits, 1.3 * pr.norm(x.sum(0), w["final.norm"], eps) @ w["head"].T)
    # keys have root mean square one, values do not
    assert torch.allclose((kv[0] ** 2).mean(-1), torch.ones(6, 1, dtype=F64), atol=1e-3)


def test_every_mechanism_counts_in_the_tests_weights():
    """The plain logits change by far more than the GPU tests' limit when a mechanism is left out of the plain
    implementation: otherwise those comparisons would not notice its absence in the engine."""
    cfg = rc.MIXED_A
    w = {n: torch.tensor(a, dtype=F64) for n, a in rc._tensors(cfg, 5).items()}
    toks = torch.randint(0, cfg["vocab"], (80,), generator=torch.Generator().manual_seed(9)).tolist()
    ref = pr.forward(cfg, w, toks)

    def differs(cfg2=cfg, w2=w):
        d = pr.forward(cfg2, w2, toks) - ref
        d = d - d.mean(-1, keepdim=True)
        return (d.pow(2).mean(-1).sqrt() / ref.std(-1)).max().item()

    def without(edit):
        c = copy.deepcopy(cfg)
        edit(c)
        return c

    for name, edit in (("chunk one longer", lambda c: c["layers"][0]["mixer"]["mask"].update(size=20)),
                       ("the reader's own chunk", lambda c: c["layers"][2]["mixer"]["mask"].update(size=19)),
                       ("the reader's shorter chunk", lambda c: c["layers"][4]["mixer"]["mask"].update(size=50)),
                       ("limit", lambda c: c["layers"][0]["mlp"].update(limit=50.0)),
                       ("logit scale", lambda c: c.update(logit_scale=1.0))):
        assert differs(cfg2=without(edit)) > 0.02, name
    for name, key, val in (("bias of k", "l0.mix.k.b", lambda t: t * 0), ("bias of v", "l0.mix.v.b", lambda t: t * 0),
                           ("earliest tap of q", "l0.mix.q.conv", lambda t: torch.cat([t[:, :1] * 0, t[:, 1:]], 1)),
                           ("earliest tap of v", "l0.mix.v.conv", lambda t: torch.cat([t[:, :1] * 0, t[:, 1:]], 1)),
                           ("direction of the mixing", "l1.hc2.mix", lambda t: t.T), ("norm of the embedding", "embed.norm", lambda t: t * 0 + 1),
                           ("order of the streams", "l1.hc1.in", lambda t: t.flip(0))):
        w2 = dict(w)
        w2[key] = val(w[key])
        assert differs(w2=w2) > 0.02, name
    keep = pr.sink_attend
    try:
        pr.sink_attend = lambda s, m, v: torch.einsum("hij,hjd->ihd", torch.softmax(s.masked_fill(~m.unsqueeze(0), -math.inf), -1), v)
        assert differs() > 0.02, "sink"
    finally:
        pr.sink_attend = keep

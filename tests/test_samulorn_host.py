"""Samulorn without a GPU: configuration (keys, errors, round trip), the model as a specification, checkpoint names and shapes, cache
and state places, what the parts make of their weights, and the plain implementation's own consistency (closed forms of its
mechanisms)."""
import copy
import math
import random

import pytest
import torch

import plain_samulorn as ps
import samulorn_configs as sc
from llm_steadyinfer_b200.config import ConfigError, config_from_dict, load_config
from llm_steadyinfer_b200.csrc import ops
from llm_steadyinfer_b200.models import Model
from llm_steadyinfer_b200.parts import NormedDelta
from llm_steadyinfer_b200.weights.loader import load_weights_into

F64 = torch.float64


def test_configuration_round_trip_and_spec():
    cfg = config_from_dict(sc.MIXED_A)
    assert config_from_dict(cfg.to_dict()) == cfg
    spec = cfg.model_spec()
    assert spec.order == [0, 1, 2, 1, 2, 3, 4] and spec.vocab_size == 331 and spec.hidden_size == 96
    assert spec.tie_word_embeddings and spec.embedder.params["scale"] == 2.0 and spec.final_norm.kind == "dynamic_tanh"
    assert spec.token_side.dim == 12 and spec.token_side.eps == 1e-5 and all(l.token_side_prefix == "side." for l in spec.layers)
    assert all(l.arrangement == "sandwich" and l.mixer_norm.kind == "dynamic_tanh" and l.mixer_post_norm.kind == "dynamic_tanh" for l in spec.layers)
    d = spec.layers[0].mixer
    assert d.kind == "channel_delta" and d.params["num_heads"] == 6 and d.params["num_kv_heads"] == 2 and d.params["conv_taps"] == 3
    m = spec.layers[1].mixer
    assert m.kind == "mixer_pair" and m.params["left_scale"] == 0.8 and m.params["right_scale"] == 1.4
    left, right = m.params["left"], m.params["right"]
    assert left["kind"] == "attention" and left["params"]["biases"] and left["params"]["rot_interleaved"] and left["params"]["qk_norm"] == {"eps": 1e-5}
    assert left["position"]["params"]["scaling"]["rope_type"] == "llama3" and right["kind"] == "gated_recurrence" and right["params"]["blocks"] == 3
    ff = spec.layers[1].feed_forward.params
    assert ff["groups"] == {"count": 5, "keep": 3} and ff["renorm"] and ff["scale"] == 2.5 and ff["choice_bias"] == "correction" and ff["activation"] == "silu_glu"
    assert spec.layers[2].feed_forward is None and spec.layers[3].feed_forward.params["groups"] is None
    bare = config_from_dict({k: v for k, v in sc.ONLY_DELTA.items() if k != "embedding"})
    assert bare.embedding_scale == 1.0 and bare.model_spec().token_side is None and bare.model_spec().order == [0]


def _at(d, *path):
    for p in path:
        d = d[p]
    return d


@pytest.mark.parametrize("edit,word", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d["token_side"].update(dim=0), "dim"),
    (lambda d: d["embedding"].update(scale="big"), "scale"),
    (lambda d: d.update(layers=[]), "layers"),
    (lambda d: d["layers"][0].update(type="attention"), "type"),
    (lambda d: d["layers"][0].pop("mixer"), "mixer"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"].pop("left"), "left"),
    (lambda d: _at(d, "layers", 1, "mixer", "left").pop("scale"), "scale"),
    (lambda d: _at(d, "layers", 1, "mixer", "left", "rot").update(dims=23), "dims"),
    (lambda d: _at(d, "layers", 1, "mixer", "left", "rot", "scaling").pop("original"), "original"),
    (lambda d: _at(d, "layers", 1, "mixer", "right").update(blocks=5), "blocks"),
    (lambda d: _at(d, "layers", 1, "mixer", "right").pop("width"), "width"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda d: _at(d, "layers", 1, "mlp", "router").update(top=11), "top"),
    (lambda d: _at(d, "layers", 1, "mlp", "router", "groups").update(count=4), "groups"),
    (lambda d: _at(d, "layers", 1, "mlp", "router", "groups").update(keep=1), "groups"),
    (lambda d: d["loop"].update(stop=9), "loop"),
    (lambda d: d["loop"].pop("times"), "times"),
])
def test_configuration_errors_name_the_key(edit, word):
    d = copy.deepcopy(sc.MIXED_A)
    edit(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


@pytest.mark.parametrize("name", sorted(sc.CONFIGS))
def test_checkpoint_names_and_shapes(name, tmp_path):
    folder = sc.write_folder(str(tmp_path / "m"), sc.CONFIGS[name], 3)
    model = Model(load_config(folder), torch.float32, "cpu")
    want = {n: a.shape for n, a in sc._tensors(sc.CONFIGS[name], 0).items()}
    assert model.weight_shapes() == want
    load_weights_into(model, folder)
    assert model.capturable() and model.lm_head is model.embed


def test_cache_and_state_places(tmp_path):
    model = Model(config_from_dict(sc.MIXED_A), torch.float32, "cpu")
    needs, states = model.cache_places()
    assert len(needs) == 8 and [n is not None for n in needs] == [False, True, False, True, False, True, False, False]
    assert (needs[1].num_kv_heads, needs[1].head_dim, needs[1].v_dim, needs[1].window, needs[1].chunk) == (2, 24, 16, None, None)
    # the delta rule: the heads' matrices, then the last inputs of the convolution over q, k and v
    assert states[0].shape == (6 * ops.delta_state_floats(24, 16) + 2 * (48 + 48 + 96),)
    # the pair: the left side's convolution, then (on a 16-byte boundary) the recurrence and its convolution
    assert states[1].shape == (3 * (96 + 48 + 32) + 72 + 3 * 72,)
    left, right = model.blocks[3].mixer.subs
    assert left.state_need() is None and model.blocks[3].mixer.state_need() == right.state_need()      # one tap: nothing to remember
    odd = Model(config_from_dict(sc.ODD), torch.float32, "cpu")
    assert all(s is None or s.shape[0] % 4 == 0 for s in odd.cache_places()[1])


def test_what_the_parts_make_of_their_weights(tmp_path):
    folder = sc.write_folder(str(tmp_path / "m"), sc.MIXED_A, 4)
    model = Model(load_config(folder), torch.float32, "cpu")
    load_weights_into(model, folder)
    _, w = ps.read_model_folder(folder)
    b = model.blocks[0]
    n = b.mixer_norm
    assert torch.equal(n.weight.double(), w["l0.norm1"]) and torch.equal(n.bias.double(), w["l0.norm1.b"]) and n.alpha == w["l0.norm1.alpha"].item()
    m = b.mixer                                                   # [q | k | v | b | a1 | g1], pieces from multiples of 8 on
    assert m.b_off == 192 and m.a_cols == (200, 216) and m.g_cols == (216, 232) and m.w_in.shape == (232, 96)
    assert torch.equal(m.w_in[200:210].double(), w["l0.mix.a1"]) and not m.w_in[198:200].any() and not m.w_in[210:216].any()
    assert torch.equal(m.w_a2[:, :10].double(), w["l0.mix.a2"]) and not m.w_a2[:, 10:].any()
    pair = model.blocks[1].mixer
    left, right = pair.subs
    # one input product and one output product for both sides; the left side's scale sits in its values' taps, the right one's is applied later
    assert torch.equal(pair.w_in[:96].double(), w["l1.mix.left.q"]) and torch.equal(pair.w_in[176:176 + 72].double(), w["l1.mix.right.y"])
    assert torch.equal(pair.w_o[:, :64].double(), w["l1.mix.left.o"]) and torch.equal(pair.w_o[:, 64:].double(), w["l1.mix.right.o"])
    assert torch.allclose(left.qkv_taps[:, 144:].double(), 0.8 * w["l1.mix.left.v.conv"].T, rtol=1e-6)
    assert torch.equal(left.qkv_taps[:, :144].double(), torch.cat([w["l1.mix.left.q.conv"], w["l1.mix.left.k.conv"]]).T)
    assert pair.scales == (1.0, 1.4)
    assert torch.allclose(right.rate.double(), 8.0 * torch.nn.functional.softplus(w["l1.mix.right.lam"]), rtol=1e-6)
    assert torch.equal(right.w_gates[:, :24].double(), w["l1.mix.right.ra"]) and torch.equal(right.w_gates[:, 24:].double(), w["l1.mix.right.ri"])
    assert torch.allclose(left.rot[0].double(), ps.frequencies(sc.MIXED_A["layers"][1]["mixer"]["left"]["rot"]), rtol=1e-6)
    s = model.blocks[4].token_side
    assert torch.equal(s.table.double(), w["side.embed"][:, 48:60]) and s.pad == 16 and not s.gate[12:].any() and not s.proj[:, 12:].any()


def test_a_pending_result_with_either_norm_has_a_plain_value(tmp_path):
    """What hooks see of a pending result: the norm behind the sublayer applied, whatever its kind."""
    folder = sc.write_folder(str(tmp_path / "m"), sc.MIXED_A, 4)
    model = Model(load_config(folder), torch.float32, "cpu")
    load_weights_into(model, folder)
    _, w = ps.read_model_folder(folder)
    x = torch.randn(5, 96)
    got = NormedDelta(x, model.blocks[0].mixer_post_norm).value()
    assert torch.allclose(got.double(), ps.tanh_norm(x.double(), w, "l0.norm1b"), atol=1e-5)
    got = NormedDelta(x, model.blocks[0].token_side.norm, torch.ones(96)).value()
    assert torch.allclose(got.double(), ps.over_rms(x.double() + 1.0, 1e-5) * w["l0.side.norm"], atol=1e-5)


def test_random_weights_need_a_rank():
    from llm_steadyinfer_b200.weights.random_init import random_tensors
    d = copy.deepcopy(sc.ONLY_DELTA)
    t = random_tensors(Model(config_from_dict(d), torch.float32, "cpu"), 0, torch.float32)
    assert t["l0.mix.a1"].shape == (12, 64) and abs(t["l0.norm1.alpha"].item() - 1) < 0.7 and t["l0.norm1.b"].abs().max() < 0.2
    d["layers"][0]["mixer"].pop("rank")
    with pytest.raises(ValueError, match="a1|a2|g1|g2"):
        random_tensors(Model(config_from_dict(d), torch.float32, "cpu"), 0, torch.float32)


def test_routed_feed_forward_refuses_groups_that_do_not_fit():
    from llm_steadyinfer_b200.parts.moe import RoutedMLP
    base = {"hidden_size": 16, "intermediate_size": 8, "experts": 12, "top": 3, "choice_bias": "correction", "activation": "silu_glu"}
    RoutedMLP(dict(base, groups={"count": 4, "keep": 1}), torch.float32, "cpu")
    for bad in ({"count": 5, "keep": 2}, {"count": 4, "keep": 5}, {"count": 6, "keep": 1}):
        with pytest.raises(ValueError):
            RoutedMLP(dict(base, groups=bad), torch.float32, "cpu")
    with pytest.raises(ValueError):
        RoutedMLP(dict(base, choice_bias=None, groups={"count": 4, "keep": 2}), torch.float32, "cpu")


# ---- the plain implementation against closed forms ------------------------------------------------------------------

def test_plain_delta_rule_with_equal_decays_is_a_decaying_projection():
    """With one key at every step and beta 1 the state holds the last value alone; with orthogonal keys the read-out finds each value with
    its own key channel's decay."""
    T, dk, dv = 6, 4, 3
    v = torch.randn(T, dv, dtype=F64)
    k = torch.zeros(T, dk, dtype=F64)
    k[:, 1] = 1.0
    o = ps.delta_head(k, k, v, torch.ones(T, dtype=F64), torch.full((T, dk), 0.7, dtype=F64))
    assert torch.allclose(o, v)
    k = torch.eye(dk, dtype=F64)
    q = torch.ones(dk, dk, dtype=F64)
    g = torch.tensor([0.9, 0.5, 0.8, 0.3], dtype=F64)
    o = ps.delta_head(q, k, v[:dk], torch.ones(dk, dtype=F64), g.expand(dk, dk))
    want = torch.stack([sum(g[i] ** (t - i) * v[i] for i in range(t + 1)) for t in range(dk)])
    assert torch.allclose(o, want)


def test_plain_linear_recurrence_closed_form():
    """Gates held open by their biases: a constant decay a, so S_t = sum a^(t - j) sqrt(1 - a^2) u_j."""
    T, W = 7, 6
    w = {"ra": torch.zeros(2, 3, 3, dtype=F64), "ra.b": torch.full((2, 3), 40.0, dtype=F64), "ri": torch.zeros(2, 3, 3, dtype=F64),
         "ri.b": torch.full((2, 3), 40.0, dtype=F64), "lam": torch.linspace(-4, -1, W, dtype=F64)}
    u = torch.randn(T, W, dtype=F64)
    a = torch.exp(-8.0 * torch.nn.functional.softplus(w["lam"]))
    want = torch.stack([sum(a ** (t - j) * torch.sqrt(1 - a * a) * u[j] for j in range(t + 1)) for t in range(T)])
    assert torch.allclose(ps.gated_unit(u, w, "", 2), want)


def test_plain_choice_by_groups():
    """The best expert of a group that is left out is not chosen, scores may be negative, and the correction moves the choice alone."""
    router = {"top": 2, "groups": {"count": 3, "keep": 1}}
    s = torch.tensor([0.9, 0.1, 0.6, 0.55, 0.2, 0.2], dtype=F64)
    zero = torch.zeros(6, dtype=F64)
    assert ps.choose(s, zero, router) == [2, 3]
    assert ps.choose(s, zero - 5.0, router) == [2, 3]
    assert ps.choose(s, torch.tensor([0.0, 0.3, 0, 0, 0, 0], dtype=F64), router) == [0, 1]
    assert sorted(ps.choose(s, zero, {"top": 2})) == [0, 2]
    assert ps.choice_margin(s, zero, router) == pytest.approx(0.15)
    assert ps.choice_margin(s, zero, {"top": 2}) == pytest.approx(0.05)


def test_plain_frequencies_and_rotation():
    rot = {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}}
    f, g = ps.frequencies({"base": 10000.0, "dims": 8}), ps.frequencies(rot)
    wave = 2 * math.pi / f
    assert wave[0] < 25 and torch.equal(g[0], f[0]) and wave[3] > 100 and g[3] == f[3] / 4
    assert f[1] / 4 < g[1] < f[1]                                # between the edges
    x = torch.randn(5, 2, 10, dtype=F64)
    y = ps.rotate(x, rot)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 8:], x[..., 8:])
    assert torch.allclose((y * y).sum(-1), (x * x).sum(-1))
    assert torch.allclose(y[3, 0, 0], x[3, 0, 0] * math.cos(3.0) - x[3, 0, 1] * math.sin(3.0))


def test_plain_is_causal_and_every_mechanism_shows(tmp_path):
    """Changing a token changes no earlier row; taking a mechanism out changes the logits (so a test against them would see it gone)."""
    folder = sc.write_folder(str(tmp_path / "m"), sc.MIXED_A, 5)
    cfg, w = ps.read_model_folder(folder)
    toks = [random.Random(1).randrange(331) for _ in range(24)]
    base = ps.forward(cfg, w, toks)
    other = list(toks)
    other[20] = (other[20] + 7) % 331
    assert torch.equal(ps.forward(cfg, w, other)[:20], base[:20])
    far = list(toks)
    far[1] = (far[1] + 7) % 331
    assert (ps.forward(cfg, w, far)[-1] - base[-1]).abs().max() > 1e-2
    for name, value in (("l0.mix.dt_bias", -20.0), ("l0.mix.q.conv", 1.0), ("l1.mix.left.q.b", 0.0), ("l1.mix.left.v.conv", 0.5),
                        ("l1.mix.right.lam", -20.0), ("l1.mix.right.conv.b", 0.0), ("l1.mix.right.ri.b", 0.0), ("l1.mlp.correction", 0.0),
                        ("l2.side.norm", 0.0), ("l3.norm2b.b", 0.0), ("l4.norm1.alpha", 0.1)):
        changed = dict(w)
        changed[name] = torch.full_like(w[name], value)
        assert (ps.forward(cfg, changed, toks)[-1] - base[-1]).abs().max() > 1e-2, name

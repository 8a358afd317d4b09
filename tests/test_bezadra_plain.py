"""The Bezadra design without a GPU: configuration reading and refusals, tensor names, what the cache keeps, the rotation's
frequencies, and the plain implementation's own mechanisms and sensitivity."""
import numpy as np
import pytest
import torch

import bezadra_helpers as bh
import plain_bezadra as plain


def _model(cfg):
    from llaisys_b200.config import config_from_dict
    from llaisys_b200.engine.model import DecoderModel
    from llaisys_b200.parts import BuildEnv
    return DecoderModel(config_from_dict(cfg).to_spec(), BuildEnv(torch.float32, torch.device("cpu")))


def test_configuration_is_read_and_turned_into_a_spec():
    from llaisys_b200.config import config_from_dict
    c = config_from_dict(bh.CONFIGS["P"])
    assert (c.vocab, c.width, c.embed_scale, c.logit_scale, c.loop) == (211, 64, 3.0, 0.5, (1, 3, 3))
    spec = c.to_spec()
    assert [e.layer for e in spec.order] == [0, 1, 2, 1, 2, 1, 2, 3] and [e.opens_pass for e in spec.order] == [None, 0, None, 1, None, 2, None, None]
    assert spec.reentry.kind == "embedding_projection" and spec.reentry.params["passes"] == 3 and spec.head.params["tied_to"] == "embed"
    d, a = spec.layers[0].sublayers[0], spec.layers[1].sublayers[0]
    assert (d.part.kind, d.part.params["num_kv_heads"], d.part.params["taps"], d.norm.kind) == ("channel_delta_rule", 2, 4, "layer_norm")
    assert (a.part.kind, a.part.params["softcap"], a.part.params["sink"], a.part.params["gate"]) == ("windowed_sink_attention", 6.0, "learned", "elements")
    assert a.part.params["position"].params["wave"] == {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64.0}
    assert [len(l.sublayers) for l in spec.layers] == [2, 2, 1, 2] and spec.layers[3].sublayers[1].part.params["limit"] == float("inf")
    q = config_from_dict(bh.CONFIGS["Q"])
    assert (q.loop, q.logit_scale, q.embed_scale, q.to_spec().reentry) == (None, 1.0, 1.0, None) and q.to_dict() == bh.CONFIGS["Q"]
    assert q.to_spec().layers[0].sublayers[0].part.params["position"] is None and not q.mixers[0].softcap


def test_what_may_be_left_out():
    from llaisys_b200.config import config_from_dict

    def bare(c):
        for l in c["layers"]:
            l["mixer"].pop("kv_heads")
            l["mixer"].pop("vdim")
    c = config_from_dict(bh.variant(bh.CONFIGS["P"], bare))
    assert [(m.kv_heads, m.vdim) for m in c.mixers] == [(4, 16), (4, 16), (2, 24), (2, 24)]


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=11), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "dense"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0), "limit"),
    (lambda c: c["layers"][0].update(type="gla"), "mixers"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configurations_that_cannot_be_are_refused(edit, text):
    from llaisys_b200.config import ConfigError, config_from_dict
    with pytest.raises(ConfigError, match=text):
        config_from_dict(bh.variant(bh.CONFIGS["P"], edit))


def test_heads_the_kernels_do_not_take_are_refused_when_the_model_is_built():
    from llaisys_b200.kernels import KernelError
    for edit in (lambda c: c["layers"][0]["mixer"].update(dim=257), lambda c: c["layers"][0]["mixer"].update(vdim=300),
                 lambda c: c["layers"][3]["mixer"].update(vdim=260)):
        with pytest.raises(KernelError):
            _model(bh.variant(bh.CONFIGS["P"], edit))


def test_tensor_names_and_shapes():
    t = _model(bh.CONFIGS["P"]).expected_tensors()
    want = {"embed": (211, 64), "final.norm": (64,), "loop.in": (64, 128), "loop.step": (3, 64), "l0.norm1": (64,), "l0.mix.q": (32, 64),
            "l0.mix.q.conv": (32, 4), "l0.mix.v": (96, 64), "l0.mix.v.conv": (96, 4), "l0.mix.b": (4, 64), "l0.mix.A_log": (4,),
            "l0.mix.norm": (24,), "l0.mix.dt_bias": (64,), "l0.mix.o": (64, 96), "l0.mlp.gate": (40, 64), "l0.mlp.down": (64, 40),
            "l1.mix.q": (64, 64), "l1.mix.k": (32, 64), "l1.mix.v": (48, 64), "l1.mix.sink": (4,), "l1.mix.g": (96, 64), "l1.mix.o": (64, 96)}
    for name, shape in want.items():
        assert tuple(t[name].shape) == shape, name
    assert t["l0.mix.a1"].free == t["l0.mix.g1"].free == (0,) and t["l0.mix.a2"].free == t["l0.mix.g2"].free == (1,)
    assert "head" not in t and "l2.mlp.gate" not in t and "l0.norm2" not in t
    assert not any(n.startswith("loop") for n in _model(bh.CONFIGS["Q"]).expected_tensors())


def test_bottlenecks_of_any_size_and_a_pair_that_does_not_fit(tmp_path):
    from llaisys_b200.models.cpu_model import CpuModel
    cfg = bh.config(60, 32, [bh.delta(2, 1, 8, 12, 3, bh.dense(16))])
    rng = np.random.default_rng(0)

    def ranks(t):
        t["l0.mix.a1"], t["l0.mix.a2"] = (torch.from_numpy(rng.normal(size=s) * 0.3).bfloat16() for s in ((5, 32), (16, 5)))
        t["l0.mix.g1"], t["l0.mix.g2"] = (torch.from_numpy(rng.normal(size=s) * 0.3).bfloat16() for s in ((11, 32), (24, 11)))
    folder = bh.make_folder(tmp_path / "a", cfg, seed=1, gain=4.0, edit=ranks)
    toks = bh.random_requests(cfg, [20], seed=1)[0]
    assert np.abs(CpuModel.from_folder(folder).step(toks) - bh.Oracle(folder).logits(toks)).max() < 2e-4
    from llaisys_b200.weights import FolderSource, load_weights
    load_weights(_model(cfg), FolderSource(folder))
    folder = bh.make_folder(tmp_path / "b", cfg, seed=1, gain=4.0, edit=lambda t: t.update({"l0.mix.a2": torch.zeros((16, 7)).bfloat16()}))
    with pytest.raises(ValueError, match="do not fit"):
        load_weights(_model(cfg), FolderSource(folder))


def test_what_the_cache_keeps():
    from llaisys_b200.cache.kv import CacheConfig, PagedCache
    m = _model(bh.CONFIGS["P"])
    # run order: layer 0, then (1, 2) three times, then 3; a recurrent layer is two users of the fixed-size state
    assert [len(u) for u in m.call_all_users] == [2, 1, 2, 1, 2, 1, 2, 1]
    needs, states = m.kv_needs(), m.state_sizes()
    assert states[:5] == [4 * 16 * 24, 3 * (2 * 2 * 16 + 4 * 24), 0, 2 * 24 * 16, 3 * (2 * 2 * 24 + 2 * 16)]
    assert needs[0] is None and needs[2].window is None and (needs[2].key_dim, needs[2].value_dim) == (16, 24)
    c = PagedCache(needs, m.cache_of(), states, CacheConfig(max_tokens=64 * 12, max_seqs=2), torch.float32, "cpu")
    assert c.group_keys == [(2, 16, 24, None, 0), (1, 24, 8, None, 0)] and len(c.state) == 8
    assert _model(bh.CONFIGS["Q"]).state_sizes()[3:5] == [2 * 33 * 35, 0]                # one tap: nothing to carry


# ----------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("wave", [None, (4.0, 1.0, 4.0, 64), (8.0, 2.0, 2.0, 32), (3.0, 1.0, 1.5, 1000), (0.5, 1.0, 8.0, 50)])
def test_frequencies_rescaled_by_wavelength(wave):
    from llaisys_b200.parts.rope import wavelength_frequencies
    r = bh.rot(24, 2000.0, wave)
    want = plain.frequencies(r)
    got = wavelength_frequencies(24, 2000.0, r.get("scaling")).numpy()
    assert np.allclose(got, want, rtol=1e-12, atol=0)
    f = 2000.0 ** (-2.0 * np.arange(12) / 24)
    if wave is None:
        assert np.allclose(want, f)
        return
    factor, low, high, original = wave
    turns = original * f / (2 * np.pi)
    assert np.allclose(want[turns > high], f[turns > high]) and np.allclose(want[turns < low], f[turns < low] / factor)
    between = (turns < high) & (turns > low)
    lo, hi = np.minimum(f, f / factor), np.maximum(f, f / factor)
    assert ((want > lo) & (want < hi))[between].all()


def test_rotation_tables_follow_the_frequencies():
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import BuildEnv, build_part
    r = bh.rot(12, 2000.0, (4.0, 1.0, 4.0, 64))
    part = build_part("position", PartSpec("rope_leading", {"head_dim": 16, "dims": 12, "base": 2000.0, "wave": r["scaling"]}),
                      BuildEnv(torch.float32, torch.device("cpu")))
    cos, sin = part.leading_tables(200)
    ang = np.arange(200)[:, None] * plain.frequencies(r)[None, :]
    assert np.abs(cos[:200].numpy() - np.cos(ang)).max() < 1e-6 and np.abs(sin[:200].numpy() - np.sin(ang)).max() < 1e-6
    plain_part = build_part("position", PartSpec("rope_leading", {"head_dim": 16, "dims": 12, "base": 2000.0}), BuildEnv(torch.float32, torch.device("cpu")))
    assert np.abs(plain_part.leading_tables(200)[0][:200].numpy() - cos[:200].numpy()).max() > 0.1       # tables of their own


# ----------------------------------------------------------------------------- the plain implementation itself
def test_short_convolution():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    y = plain.short_conv(x, w)
    assert y[:, 1].tolist() == x[:, 1].tolist() and y[0, 0] == 0 and y[1, 0] == 200 and y[3, 0] == 100 * 6 + 10 * 4 + 2
    assert np.array_equal(plain.short_conv(x[:1], w), x[:1] * w[:, 2])


def test_delta_rule_stores_replaces_and_forgets():
    k = np.zeros((4, 1, 3))
    k[0, 0, 0] = k[1, 0, 1] = k[2, 0, 0] = k[3, 0, 2] = 1.0
    q = np.ones((4, 1, 3))
    v = np.array([[[2.0, 3.0]], [[5.0, 7.0]], [[11.0, 13.0]], [[0.0, 0.0]]])
    one, beta = np.ones((4, 1, 3)), np.ones((4, 1))
    o = plain.delta_rule(q, k, v, one, beta)
    # the read-out sees the token's own write; a second write under the same key replaces the first
    assert o[:, 0].tolist() == [[2, 3], [7, 10], [16, 20], [16, 20]]
    g = one.copy()
    g[3, 0, 0] = 0.0                                        # what key channel 0 held is gone
    assert plain.delta_rule(q, k, v, g, beta)[3, 0].tolist() == [5, 7]
    assert plain.delta_rule(q, k, v, one, beta * 0.5)[2, 0].tolist() == [8.5, 10.75]


def test_sink_softmax_and_cap():
    w = plain.sink_softmax(np.zeros((3, 3)), np.log(2.0))
    assert np.allclose(w[2], 1 / 5) and np.allclose(w[0], [1 / 3, 0, 0])
    assert np.allclose(plain.capped(np.array([0.01, 1e9, -1e9]), 5.0), [0.01, 5.0, -5.0], atol=1e-6) and plain.capped(7.0, None) == 7.0


def test_layer_norm_and_unit_vectors():
    x = np.array([[1.0, 2.0, 6.0]])
    assert np.allclose(plain.layer_norm(x, np.array([1.0, 1.0, 2.0]), 0.0), (x - 3) / np.sqrt(14 / 3) * [1, 1, 2])
    assert np.allclose(plain.unit(np.array([3.0, 4.0])), [0.6, 0.8]) and np.isclose(plain.unit(np.array([1e-3, 0.0]))[0], 2 ** -0.5)


def test_feed_forward_clamps():
    one = np.ones((1, 1))
    y = lambda g, u, limit=1.5: plain.feed_forward(np.array([[1.0]]), {"gate": one * g, "up": one * u, "down": one}, {"limit": limit})[0, 0]
    assert np.isclose(y(9.0, 0.0), 1.5 * plain.sigmoid(1.702 * 1.5)) and np.isclose(y(1.0, 7.0), plain.sigmoid(1.702) * 2.5)
    assert np.isclose(y(1.0, -7.0), plain.sigmoid(1.702) * -0.5) and np.isclose(y(-9.0, 0.0), -9.0 * plain.sigmoid(1.702 * -9.0))
    assert np.isclose(y(9.0, 7.0, None), 9.0 * plain.sigmoid(1.702 * 9.0) * 8.0)


SENSITIVE = [
    ("the cap", lambda c: c["layers"][1]["mixer"].update(softcap=6.6), 1),
    ("the scale of the scores", lambda c: c["layers"][1]["mixer"].update(scale=0.27), 0),
    ("the rescaling's factor", lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=4.4), 1),
    ("the rescaling's lower edge", lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=1.3), 1),
    ("the rescaling's upper edge", lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=3.0), 1),
    ("the rescaling's original length", lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(original=70), 1),
    ("the rotated dimensions", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), 1),
    ("the feed-forward's limit", lambda c: c["layers"][0]["mlp"].update(limit=0.9), 0),
    ("the number of passes", lambda c: c["loop"].update(times=2), 0),
    ("the embedding's scale", lambda c: c["embedding"].update(scale=3.3), 0),
    ("the logit scale", lambda c: c.update(logit_scale=0.51), 0),
    ("the norm's eps", lambda c: c["norm"].update(eps=1e-1), 0),
]


@pytest.fixture(scope="module")
def p_model(tmp_path_factory):
    folder = bh.make_folder(tmp_path_factory.mktemp("p"), bh.CONFIGS["P"], seed=3, gain=40.0)
    o = bh.Oracle(folder)
    return o.config, {k: np.asarray(v, dtype=np.float64) for k, v in o.weights.items()}


@pytest.mark.parametrize("what, edit, first", SENSITIVE, ids=[s[0] for s in SENSITIVE])
def test_every_constant_moves_the_logits_from_where_it_should(p_model, what, edit, first):
    """A constant that is off by some per cent moves the logits by far more than any tolerance of the GPU tests, and leaves
    bit-equal the positions it cannot reach: those before `first`."""
    cfg, w = p_model
    toks = bh.random_requests(cfg, [60], seed=1)[0]
    a = plain.forward(cfg, w, toks)[0]
    moved = np.abs(a - plain.forward(bh.variant(cfg, edit), w, toks)[0]).max(axis=1)
    assert moved[first:].max() > 3e-3, (what, moved.max())
    assert first == 0 or what == "the cap" or moved[:first].max() == 0.0, (what, moved[:first].max())


def test_each_tensor_of_a_layer_matters(p_model):
    cfg, w = p_model
    toks = bh.random_requests(cfg, [50], seed=2)[0]
    a = plain.forward(cfg, w, toks)[0]
    for name in w:
        w2 = dict(w, **{name: w[name] * 1.2 + 0.05})
        assert np.abs(plain.forward(cfg, w2, toks)[0] - a).max() > 1e-3, name


def test_the_first_token_reaches_the_last_position_through_either_mixer():
    for layer in (bh.delta(2, 1, 8, 8, 4), bh.attention(2, 1, 8, 8, softcap=9.0, rotation=bh.rot(8))):
        import tempfile
        cfg = bh.config(50, 32, [layer])
        with tempfile.TemporaryDirectory() as tmp:
            o = bh.Oracle(bh.make_folder(tmp, cfg, seed=2, gain=20.0, edit=lambda t: t.update({k: v - 4 for k, v in t.items() if k.endswith("A_log")})))
            toks = np.random.default_rng(4).integers(0, 49, size=40).tolist()
            moved = np.abs(o.logits(toks) - o.logits([49] + toks[1:])).max(axis=1)
            assert moved[-1] > 1e-4, layer["type"]


@pytest.mark.parametrize("name", ["P", "Q", "R"])
def test_cpu_model_against_the_plain_implementation(tmp_path, name):
    """The package's CPU model (float32 operators, a cache, the prompt and then single tokens) against the plain float64
    evaluation of whole sequences: whole prompts, and the same tokens fed in portions down to single ones."""
    from llaisys_b200.models.cpu_model import CpuModel
    cfg = bh.CONFIGS[name]
    folder = bh.make_folder(tmp_path, cfg, seed=4, gain=40.0)
    toks = bh.random_requests(cfg, [90], seed=7)[0]
    ref = bh.Oracle(folder).logits(toks)
    model = CpuModel.from_folder(folder)
    assert np.abs(model.step(toks) - ref).max() < 2e-4
    model.reset()
    got = np.concatenate([model.step(toks[:70]), model.step(toks[70:72])] + [model.step([t]) for t in toks[72:]])
    assert np.abs(got - ref).max() < 2e-4

"""The Zupitar design without a GPU: configuration reading and refusals, tensor names, what the cache keeps, and the plain
implementation's own mechanisms and sensitivity."""
import numpy as np
import pytest
import torch

import plain_zupitar as plain
import zupitar_helpers as zh


def _model(cfg):
    from llaisys_b200.config import config_from_dict
    from llaisys_b200.engine.model import DecoderModel
    from llaisys_b200.parts import BuildEnv
    return DecoderModel(config_from_dict(cfg).to_spec(), BuildEnv(torch.float32, torch.device("cpu")))


def test_configuration_is_read_and_turned_into_a_spec():
    from llaisys_b200.config import config_from_dict
    c = config_from_dict(zh.CONFIGS["P"])
    assert (c.vocab, c.width, c.eps, c.softcap) == (211, 64, 1e-5, 3.0) and c.to_dict() == zh.CONFIGS["P"]
    spec = c.to_spec()
    assert [e.layer for e in spec.order] == [0, 1, 2, 3] and spec.head.params["softcap"] == 3.0 and spec.reentry is None
    assert all(l.block == "sandwich_residual" for l in spec.layers) and [len(l.sublayers) for l in spec.layers] == [2, 2, 2, 1]
    par = spec.layers[0].sublayers[0]
    assert (par.part.kind, par.part.params["combine"], par.norm.prefix, par.post_norm.prefix) == ("parallel_mixers", "sum", "l0.norm1", "l0.norm1b")
    left, right = (b["part"] for b in par.part.params["branches"])
    assert (left.kind, left.params["values"], left.params["conv"], left.params["value_scale"]) == ("windowed_sink_attention", "keys", 4, 1.3)
    assert left.params["position"].params == {"head_dim": 16, "dims": 12, "base": 2000.0, "factor": 4.0}
    assert (right.kind, right.params["out_scale"], right.params["groups"], right.params["norm_groups"]) == ("state_space", -0.7, 2, 2)
    m = spec.layers[1].sublayers[1].part.params
    assert (m["experts"], m["identity"], m["top"], m["gate"], m["group_score"], m["groups"]) == (7, 2, 3, "softmax", "max", {"count": 3, "keep": 2})
    q = config_from_dict(zh.CONFIGS["Q"])
    assert q.softcap is None and q.ffs[1] is None and q.mixers[1].left.taps is None and q.mixers[1].left.rot is None


def test_what_may_be_left_out():
    from llaisys_b200.config import config_from_dict

    def bare(c):
        for l in c["layers"]:
            m = l["mixer"]
            for k in ("left_scale", "right_scale", "groups", "norm_groups"):
                m.pop(k, None)
            if "left" in m:
                m["left"].pop("kv_heads")
                m["left"].pop("vdim")
    c = config_from_dict(zh.variant(zh.CONFIGS["P"], bare))
    assert (c.mixers[0].left.kv_heads, c.mixers[0].left_scale, c.mixers[0].right_scale, c.mixers[1].groups, c.mixers[1].norm_groups) == (4, 1.0, 1.0, 1, 1)


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "cannot share"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=8), "values are the keys"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=11), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "cannot share"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "normed"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=10), "cannot use"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=1), "cannot give"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "cannot give"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=4), "cannot give"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "'dense' or 'moe'"),
    (lambda c: c["layers"][0].update(type="attention"), "mixers"),
    (lambda c: c.update(logit_softcap=-3), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configurations_that_cannot_be_are_refused(edit, text):
    from llaisys_b200.config import ConfigError, config_from_dict
    with pytest.raises(ConfigError, match=text):
        config_from_dict(zh.variant(zh.CONFIGS["P"], edit))


def test_sizes_the_kernels_do_not_take_are_refused_when_the_model_is_built():
    from llaisys_b200.kernels import KernelError
    for edit in (lambda c: c["layers"][1]["mixer"].update(state=257), lambda c: c["layers"][0]["mixer"]["left"].update(dim=257, vdim=257)):
        with pytest.raises(KernelError):
            _model(zh.variant(zh.CONFIGS["P"], edit))


def test_part_options_that_do_not_go_together_are_refused():
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import BuildEnv, build_part
    env = BuildEnv(torch.float32, torch.device("cpu"))
    attn = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "key_dim": 8, "value_dim": 8, "scale": 1.0}
    for extra, text in (({"conv": 4}, "values that are the keys"), ({"values": "keys", "value_dim": 4}, "one width"),
                        ({"values": "keys", "own_kv": False}, "of the layer's own"), ({"values": "queries"}, "got 'queries'"),
                        ({"value_scale": 2.0}, "constant")):
        with pytest.raises(ValueError, match=text):
            build_part("mixer", PartSpec("windowed_sink_attention", dict(attn, **extra)), env)
    moe = {"hidden_size": 32, "experts": 6, "top": 2, "expert_ff": 8, "act": "silu", "identity": 2}
    for extra in ({"gate": "softmax_chosen"}, {"renorm": True}):
        with pytest.raises(ValueError, match="renormalised"):
            build_part("ffn", PartSpec("routed_experts", dict(moe, **extra)), env)
    with pytest.raises(ValueError, match="cannot give"):
        build_part("ffn", PartSpec("routed_experts", dict(moe, gate="softmax", groups={"count": 8, "keep": 1})), env)


def test_tensor_names_and_shapes():
    t = _model(zh.CONFIGS["P"]).expected_tensors()
    want = {"embed": (211, 64), "final.norm": (64,), "head": (211, 64), "l0.norm1": (64,), "l0.norm1b": (64,), "l0.norm2b": (64,),
            "l0.mix.left.q": (64, 64), "l0.mix.left.k": (32, 64), "l0.mix.left.q.conv": (64, 4), "l0.mix.left.k.conv": (32, 4),
            "l0.mix.left.o": (64, 64), "l0.mix.right.in": (32 + 32 + 64 + 4, 64), "l0.mix.right.conv": (96, 4), "l0.mix.right.conv.b": (96,),
            "l0.mix.right.dt_bias": (4,), "l0.mix.right.A_log": (4,), "l0.mix.right.D": (4,), "l0.mix.right.norm": (32,),
            "l0.mix.right.o": (64, 32), "l0.mlp.gate": (40, 64), "l0.mlp.down": (64, 40), "l1.mix.in": (2 * 96 + 2 * 72 + 6, 64),
            "l1.mix.norm": (96,), "l1.mlp.router": (9, 64), "l1.mlp.correction": (9,), "l1.mlp.e6.gate": (24, 64), "l1.mlp.e6.down": (64, 24)}
    for name, shape in want.items():
        assert tuple(t[name].shape) == shape, name
    assert not {"l0.mix.left.v", "l1.mlp.e7.gate", "l3.norm2", "l3.mlp.gate"} & set(t)
    q = _model(zh.CONFIGS["Q"]).expected_tensors()
    assert "l1.mix.left.q.conv" not in q and tuple(q["l3.mix.left.q.conv"].shape) == (30, 1)


def test_what_the_cache_keeps():
    from llaisys_b200.cache.kv import CacheConfig, PagedCache
    m = _model(zh.CONFIGS["P"])
    # a parallel layer: token rows, the inputs of the attention's convolution, the states, the inputs of the other convolution
    assert [len(u) for u in m.call_all_users] == [4, 2, 4, 2]
    needs, states = m.kv_needs(), m.state_sizes()
    assert states[:6] == [0, 3 * 6 * 16, 4 * 16 * 8, 3 * (32 + 64), 6 * 24 * 16, 3 * (96 + 144)]
    assert (needs[0].num_kv_heads, needs[0].key_dim, needs[0].value_dim, needs[0].window) == (2, 16, 16, None) and needs[1] is needs[2] is None
    c = PagedCache(needs, m.cache_of(), states, CacheConfig(max_tokens=64 * 12, max_seqs=2), torch.float32, "cpu")
    assert len(c.state) == 10
    assert [len(u) for u in _model(zh.CONFIGS["Q"]).call_all_users] == [4, 3, 2, 3]            # no convolution, or one tap: nothing to carry


# ----------------------------------------------------------------------------- the plain implementation itself
def test_short_convolution():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    y = plain.short_conv(x, w)
    assert y[:, 1].tolist() == x[:, 1].tolist() and y[0, 0] == 0 and y[1, 0] == 200 and y[3, 0] == 100 * 6 + 10 * 4 + 2
    assert np.array_equal(plain.short_conv(x[:1], w, np.array([5.0, 7.0])), x[:1] * w[:, 2] + [5, 7])


def test_state_space_remembers_forgets_and_skips():
    x = np.array([[[2.0, 3.0]], [[0.0, 0.0]], [[0.0, 0.0]]])
    B = np.array([[[1.0, 0.0]], [[0.0, 1.0]], [[0.0, 0.0]]])
    C = np.array([[[1.0, 0.0]], [[1.0, 5.0]], [[0.0, 1.0]]])
    dt = np.array([[0.5], [1.0], [2.0]])
    y = plain.state_space(x, B, C, dt, np.array([-np.log(2.0)]), np.array([10.0]))
    assert np.allclose(y[0, 0], [1 + 20, 1.5 + 30]) and np.allclose(y[1, 0], [0.5, 0.75]) and np.allclose(y[2], 0)


def test_gate_stands_before_the_norm_of_equal_parts():
    y, z, w = np.array([[1.0, 2.0, 30.0, 40.0]]), np.array([[1.0, -1.0, 2.0, 0.5]]), np.array([1.0, 1.0, 1.0, 2.0])
    g = y * plain.silu(z)
    got = plain.gated_group_norm(y, z, w, 2, 0.0)
    assert np.allclose(got[0, :2], g[0, :2] / np.sqrt((g[0, :2] ** 2).mean())) and np.allclose(got[0, 3], 2 * g[0, 3] / np.sqrt((g[0, 2:] ** 2).mean()))


def test_router_with_groups_negative_choice_scores_and_unbiased_weights():
    z = np.log(np.array([[0.3, 0.1, 0.25, 0.05, 0.2, 0.1]]))
    c = np.array([-1.0, -1.0, -1.0, -1.0, -1.0, -0.5])
    idx, w = plain.route(z, c, {"experts": 4, "identity": 2, "top": 2})
    assert idx.tolist() == [[5, 0]] and np.allclose(w, [[0.1, 0.3]])
    idx, w = plain.route(z, c, {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert idx.tolist() == [[5, 4]] and np.allclose(w, [[0.1, 0.2]])
    # a group's score is its single largest choice score: 0.3 beats 0.25 + 0.2
    idx, _ = plain.route(np.log(np.array([[0.3, 0.01, 0.25, 0.24, 0.2 - 0.1, 0.1]])), np.zeros(6), {"experts": 6, "top": 1, "groups": {"count": 3, "keep": 1}})
    assert idx.tolist() == [[0]]


def test_an_identity_expert_returns_its_input():
    h = np.array([[1.0, -2.0]])
    w = {"router": np.array([[0.0, 0.0], [9.0, 0.0]]), "correction": np.zeros(2), "e0.gate": np.ones((1, 2)), "e0.up": np.ones((1, 2)), "e0.down": np.ones((2, 1))}
    out = plain.moe(h, w, {"router": {"experts": 1, "identity": 1, "top": 1}, "expert": {"ff": 1}})
    assert np.allclose(out, h * plain.softmax(np.array([0.0, 9.0]))[1])


def test_values_are_the_keys_before_the_rotation():
    rng = np.random.default_rng(0)
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "scale": 0.0, "conv": 2, "rot": {"dims": 4, "base": 10.0}}
    h, k = rng.normal(size=(5, 3)), rng.normal(size=(4, 3))
    w = {"q": rng.normal(size=(4, 3)), "k": k, "q.conv": rng.normal(size=(4, 2)), "k.conv": rng.normal(size=(4, 2)), "o": np.eye(4)}
    v = plain.short_conv(h @ k.T, w["k.conv"])
    assert np.allclose(plain.attention(h, w, m), np.cumsum(v, axis=0) / np.arange(1, 6)[:, None])       # flat scores: a running mean


def test_the_cap():
    assert np.allclose(plain.capped(np.array([0.01, 1e9, -1e9]), 5.0), [0.01, 5.0, -5.0], atol=1e-6) and plain.capped(7.0, None) == 7.0


SENSITIVE = [
    ("the scale of the scores", lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.27)),
    ("the stretching of positions", lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=4.4)),
    ("the rotation's base", lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=2500.0)),
    ("the rotated dimensions", lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=10)),
    ("the left scale", lambda c: c["layers"][0]["mixer"].update(left_scale=1.4)),
    ("the right scale", lambda c: c["layers"][0]["mixer"].update(right_scale=0.7)),
    ("the parts of the norm", lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=4)),
    ("the chosen experts", lambda c: c["layers"][1]["mlp"]["router"].update(top=2)),
    ("the groups", lambda c: c["layers"][1]["mlp"]["router"].pop("groups")),
    ("the kept groups", lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=1)),
    ("the cap", lambda c: c.update(logit_softcap=3.1)),
    ("the norm's eps", lambda c: c["norm"].update(eps=1e-1)),
]


@pytest.fixture(scope="module")
def p_model(tmp_path_factory):
    folder = zh.make_folder(tmp_path_factory.mktemp("p"), zh.CONFIGS["P"], seed=3, gain=40.0)
    o = zh.Oracle(folder)
    return o.config, {k: np.asarray(v, dtype=np.float64) for k, v in o.weights.items()}


@pytest.mark.parametrize("what, edit", SENSITIVE, ids=[s[0] for s in SENSITIVE])
def test_every_constant_moves_the_logits(p_model, what, edit):
    cfg, w = p_model
    toks = zh.random_requests(cfg, [60], seed=1)[0]
    moved = np.abs(plain.forward(cfg, w, toks)[0] - plain.forward(zh.variant(cfg, edit), w, toks)[0]).max()
    assert moved > 1e-2, (what, moved)


def test_each_tensor_of_a_layer_matters(p_model):
    cfg, w = p_model
    toks = zh.random_requests(cfg, [50], seed=2)[0]
    a = plain.forward(cfg, w, toks)[0]
    for name in w:
        w2 = dict(w, **{name: w[name] * 1.2 + 0.05 * np.sign(w[name])})
        if name.endswith(("left.o", "right.o", "mix.o", "down")):
            w2[name] = w[name] * np.linspace(0.5, 1.5, w[name].shape[0])[:, None]          # (a common factor meets a norm)
        assert np.abs(plain.forward(cfg, w2, toks)[0] - a).max() > 1e-3, name


def test_the_first_token_reaches_the_last_position_through_either_mixer(tmp_path):
    for i, layer in enumerate((zh.mamba2(2, 8, 8, 1, 4, 1), zh.parallel((2, 1, 8, 4, zh.rot(8)), (1, 4, 4, 1, 2, 1), (1.0, 0.0)))):
        cfg = zh.config(50, 32, [layer])
        o = zh.Oracle(zh.make_folder(tmp_path / str(i), cfg, seed=2, gain=20.0, edit=lambda t: t.update({k: v - 4 for k, v in t.items() if k.endswith("A_log")})))
        toks = np.random.default_rng(4).integers(0, 49, size=40).tolist()
        assert np.abs(o.logits(toks) - o.logits([49] + toks[1:])).max(axis=1)[-1] > 1e-4, layer["type"]


@pytest.mark.parametrize("name", ["P", "Q", "R"])
def test_cpu_model_against_the_plain_implementation(tmp_path, name):
    """The package's CPU model (float32 operators, a cache, the prompt and then single tokens) against the plain float64
    evaluation of whole sequences: whole prompts, and the same tokens fed in portions down to single ones."""
    from llaisys_b200.models.cpu_model import CpuModel
    cfg = zh.CONFIGS[name]
    folder = zh.make_folder(tmp_path, cfg, seed=4, gain=40.0)
    toks = zh.random_requests(cfg, [90], seed=7)[0]
    ref = zh.Oracle(folder).logits(toks)
    model = CpuModel.from_folder(folder)
    assert np.abs(model.step(toks) - ref).max() < 2e-4
    model.reset()
    got = np.concatenate([model.step(toks[:70]), model.step(toks[70:72])] + [model.step([t]) for t in toks[72:]])
    assert np.abs(got - ref).max() < 2e-4

"""The Bezadra design on the GPU against its plain implementation: every mechanism alone, then single layers at the places
where a fault would hide (page borders, a key far back, the first tokens, long memory), then whole models under every way
of cutting requests into steps, then generation and replay through the entry points."""
import json
import subprocess
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import bezadra_helpers as bh
import plain_bezadra as plain
from bezadra_helpers import compare as compare_bz
from helpers import build_engine, compare, run_batches, run_chunked, run_mixed, run_tail_by_one, run_whole, tolerance

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]
DEV = "cuda:0"


def _i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device=DEV)


def _f32(x):
    return torch.from_numpy(np.asarray(x)).float().to(DEV)


def _np(t):
    return t.float().cpu().numpy().astype(np.float64)


def _bf16_exact(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float64)).to(torch.bfloat16).to(torch.float64).numpy()


def _close(got, want, tol, what=""):
    err = np.abs(_np(got) - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), (what, err)


# ----------------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("H", [44, 250, 256, 1000, 1536, 2050, 3000, 4096, 5000])
@pytest.mark.parametrize("T", [1, 3, 300])
def test_layer_norm(H, T):
    """Rows far from zero mean (the mean must leave before the squares are summed), in both output types, whole and at
    chosen rows, with weights of both types."""
    from llaisys_b200 import kernels
    rng = np.random.default_rng(H + T)
    x = rng.normal(size=(T, H)) * rng.uniform(0.2, 5.0, size=(T, 1)) + rng.uniform(-20, 20, size=(T, 1))
    w = _bf16_exact(rng.uniform(0.5, 1.5, size=H))
    xd = _f32(x)
    want = plain.layer_norm(_np(xd), w, 1e-5)
    rows = rng.permutation(T)[:2]
    for wt in (_f32(w), _f32(w).bfloat16()):
        _close(kernels.layer_norm(xd, wt, 1e-5, torch.float32), want, 2e-5, "float32")
        _close(kernels.layer_norm(xd, wt, 1e-5, torch.bfloat16), want, 4e-3, "bfloat16")
        _close(kernels.layer_norm(xd, wt, 1e-5, torch.float32, rows=_i32(rows)), want[rows], 2e-5, "rows")
    assert torch.equal(xd, _f32(x))


@pytest.mark.parametrize("dtype", DTYPES)
def test_reentry_of_a_pass(dtype):
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import BuildEnv, build_part
    rng = np.random.default_rng(0)
    for T, H in ((1, 44), (5, 64), (300, 72)):
        part = build_part("reentry", PartSpec("embedding_projection", {"hidden_size": H, "passes": 2, "matrix": "in", "tensor": "step"}, "loop"),
                          BuildEnv(dtype, torch.device(DEV)))
        w, step = _bf16_exact(rng.normal(size=(H, 2 * H)) * 0.1), rng.normal(size=(2, H))
        part.load({"in": _f32(w).to(dtype), "step": _f32(step)})
        x0, x, d = (_bf16_exact(rng.normal(size=(T, H))) for _ in range(3))
        first = part.remember(_f32(x0))
        for t in range(2):
            stream = _f32(x)
            out, pending = part.forward(stream, _f32(d), first, t)
            assert pending is None and out.dtype == torch.float32
            mixed = x + d if dtype == torch.float32 else _bf16_exact(x + d)
            _close(out, np.concatenate([mixed, x0], 1) @ w.T + step[t], 1e-5 if dtype == torch.float32 else 1e-4, (T, H, t))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 7, 20, 40, 100, 300])
@pytest.mark.parametrize("limit", [0.7, float("inf")])
def test_clamped_gated_feed_forward(dtype, T, limit):
    """Every product kernel that ends in the gated activation (a few tokens in one launch, side-by-side rows, two
    accumulators, paired SMs) and the activation as a pass of its own, with gate and up values beyond the limits."""
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import BuildEnv, build_part
    for D, F in ((64, 96), (136, 200), (44, 30)):
        rng = np.random.default_rng(T + D)
        w = {"gate": _bf16_exact(rng.normal(size=(F, D)) * 0.2), "up": _bf16_exact(rng.normal(size=(F, D)) * 0.2),
             "down": _bf16_exact(rng.normal(size=(D, F)) * 0.2)}
        h = _bf16_exact(rng.normal(size=(T, D)))
        part = build_part("ffn", PartSpec("gated_mlp", {"hidden_size": D, "intermediate_size": F, "act": "swish_clamped", "limit": limit,
                                                        "alpha": 1.702, "names": {k: k for k in w}}), BuildEnv(dtype, torch.device(DEV)))
        part.load({k: _f32(v).to(dtype) for k, v in w.items()})
        x = _f32(h).to(dtype)
        want = plain.feed_forward(h, w, {"limit": None if limit == float("inf") else limit})
        tol = 2e-5 if dtype == torch.float32 else 2e-2
        _close(part.forward(x, None), want, tol, "returned")
        stream = torch.full((T, D), 3.0, device=DEV)
        if part.forward_into(x, None, stream):
            _close(stream - 3.0, want, tol, "into the stream")
        else:
            assert dtype == torch.float32 or F % 8 or D % 8


def _ctx(starts, slots, lens):
    return SimpleNamespace(tok_seq=_i32(np.repeat(np.arange(len(lens)), lens)), seq_start=_i32(starts), seq_slot=_i32(slots),
                           n_seqs=len(lens), max_new=int(max(lens)), n_new=list(lens))


def _recurrent_case(G, H, dk, dv, taps, lens, seed, rates=(-3.0, 1.5)):
    rng = np.random.default_rng(seed)
    C = 2 * G * dk + H * dv
    return dict(conv=rng.uniform(-1, 1, size=(C, taps)), a_log=rng.uniform(*rates, size=H),
                proj=[rng.normal(size=(n, C + H)) * 1.5 for n in lens], z=[rng.normal(size=(n, H * dk)) * 3 for n in lens])


def _recurrent_inputs(case, b, G, H, dk, dv):
    x, z = case["proj"][b].astype(np.float32).astype(np.float64), case["z"][b]
    n, C = len(x), 2 * G * dk + H * dv
    y = plain.silu(plain.short_conv(x[:, :C], case["conv"]))
    q = plain.unit(y[:, :G * dk].reshape(n, G, dk)) * dk ** -0.5
    k = plain.unit(y[:, G * dk:2 * G * dk].reshape(n, G, dk))
    g = np.exp(-np.exp(case["a_log"])[:, None] * plain.softplus(z).reshape(n, H, dk))
    return q, k, y[:, 2 * G * dk:].reshape(n, H, dv), g, plain.sigmoid(x[:, C:])


SHAPES = [(2, 4, 16, 24, 4), (1, 3, 6, 9, 3), (2, 2, 33, 35, 1), (1, 1, 17, 7, 6), (2, 2, 64, 64, 4), (1, 2, 128, 128, 4), (1, 1, 130, 250, 4),
          (1, 1, 256, 16, 2), (3, 3, 64, 128, 4), (1, 1, 1, 1, 4), (2, 6, 96, 40, 5), (1, 2, 16, 20, 13)]


@pytest.mark.parametrize("shape", SHAPES, ids=[str(s) for s in SHAPES])
@pytest.mark.parametrize("cuts", [(1000,), (1,), (2, 1, 3, 7, 1, 1, 40), (16, 15, 17, 1, 1000)], ids=["whole", "single", "small", "portions"])
def test_what_enters_the_recurrence_with_inputs_carried_in_slots(shape, cuts):
    """Convolution, activation, unit vectors, decays and step sizes of three sequences whose portions share steps: the
    carried inputs lie in state rows in another order than the batch, one of which was used before."""
    from llaisys_b200 import kernels
    G, H, dk, dv, taps = shape
    lens = [40, 9, 23]
    C = 2 * G * dk + H * dv
    case = _recurrent_case(G, H, dk, dv, taps, lens, seed=sum(shape))
    slots = [2, 0, 3]
    state = torch.full((4, max(1, (taps - 1) * C)), 7.0, device=DEV)
    for s in slots:
        state[s].zero_()
    conv, a_log = _f32(case["conv"].T.copy()).contiguous(), _f32(case["a_log"])
    got = [[] for _ in lens]
    at, i = [0, 0, 0], 0
    while any(at[b] < lens[b] for b in range(3)):
        n = cuts[min(i, len(cuts) - 1)]
        i += 1
        live = [b for b in range(3) if at[b] < lens[b]]
        new = [min(n + (b if n > 1 else 0), lens[b] - at[b]) for b in live]
        proj = _f32(np.concatenate([case["proj"][b][at[b]:at[b] + m] for b, m in zip(live, new)]))
        z = _f32(np.concatenate([case["z"][b][at[b]:at[b] + m] for b, m in zip(live, new)]))
        ctx = _ctx(np.concatenate([[0], np.cumsum(new)]), [slots[b] for b in live], new)
        rows, beta = kernels.delta_prep(proj, z, conv, a_log, state if taps > 1 else None, G, H, dk, dv, dk ** -0.5, ctx, fast=bool(i % 2))
        o = 0
        for b, m in zip(live, new):
            got[b].append((rows[o:o + m].clone(), z[o:o + m].clone(), beta[o:o + m].clone()))
            o += m
            at[b] += m
    assert (state[1] == 7.0).all()
    for b, n in enumerate(lens):
        q, k, v, g, be = _recurrent_inputs(case, b, G, H, dk, dv)
        rows, gg, bb = (torch.cat([x[j] for x in got[b]]) for j in range(3))
        _close(rows, np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1), 5e-6, "q, k, v")
        _close(gg, g.reshape(n, -1), 1e-6, "decays")
        _close(bb, be, 1e-6, "step sizes")


def _scan(case, lens, cuts, shape, chunked, slots=None):
    """o per sequence and the states left, of all sequences together, fed in portions."""
    from llaisys_b200 import kernels
    G, H, dk, dv, _ = shape
    slots = list(range(len(lens)))[::-1] if slots is None else slots
    state = torch.zeros((max(slots) + 1, H * dk * dv), device=DEV)
    full = [_recurrent_inputs(case, b, G, H, dk, dv) for b in range(len(lens))]
    out = [[] for _ in lens]
    at, i = [0] * len(lens), 0
    while any(at[b] < lens[b] for b in range(len(lens))):
        n = cuts[min(i, len(cuts) - 1)]
        i += 1
        live = [b for b in range(len(lens)) if at[b] < lens[b]]
        new = [min(n, lens[b] - at[b]) for b in live]
        part = [[np.asarray(x[at[b]:at[b] + m]).reshape(m, -1) for x in full[b]] for b, m in zip(live, new)]
        qkv = _f32(np.concatenate([np.concatenate(p[:3], 1) for p in part]))
        g, beta = (_f32(np.concatenate([p[j] for p in part])) for j in (3, 4))
        ctx = _ctx(np.concatenate([[0], np.cumsum(new)]), [slots[b] for b in live], new)
        o = kernels.delta_scan(qkv, g, beta, state, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, ctx.max_new, G, H, dk, dv, chunked=chunked)
        p = 0
        for b, m in zip(live, new):
            out[b].append(_np(o[p:p + m]))
            p += m
            at[b] += m
    return [np.concatenate(x) for x in out], [_np(state[s]).reshape(H, dk, dv) for s in slots], full


def _oracle_scan(full, G, H):
    q, k, v, g, beta = full
    own = np.arange(H) // (H // G)
    return plain.delta_rule(q[:, own], k[:, own], v, g, beta)


@pytest.mark.parametrize("shape", SHAPES, ids=[str(s) for s in SHAPES])
@pytest.mark.parametrize("chunked", [False, True])
def test_recurrence_against_the_oracle(shape, chunked):
    """Three sequences of unequal length in one step, and the same in portions down to single tokens: chunks that end
    anywhere, states handed on, slots in another order than the batch."""
    G, H, dk, dv, _ = shape
    lens = [70, 16, 33]
    case = _recurrent_case(*shape, lens, seed=1 + sum(shape))
    for cuts in ((1000,), (16, 1, 17, 2, 1000), (1,)) if not chunked else ((1000,), (16, 1, 17, 2, 1000), (31,)):
        out, _, full = _scan(case, lens, cuts, shape, chunked)
        for b, n in enumerate(lens):
            want = _oracle_scan(full[b], G, H).reshape(n, -1)
            err = np.abs(out[b] - want).max()
            assert err <= 5e-6 * max(1.0, np.abs(want).max()), (cuts, b, err)
    from llaisys_b200.kernels import ops
    assert ops.tc_error(DEV) == 0


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("what", ["forgets at once", "never forgets", "one key", "two keys by turns", "far write", "mixed channels"])
def test_recurrence_at_its_extremes(chunked, what):
    """Decays of zero and of one, in all channels and in some; every token under one key with a step size of almost one
    (each write replaces the last: the chunk's triangular system is as far from the identity as it gets); a single write
    hundreds of tokens before the one read-out that asks for it."""
    from llaisys_b200 import kernels
    G, H, dk, dv, n = 1, 2, 64, 48, 400
    rng = np.random.default_rng(3)
    q, k = plain.unit(rng.normal(size=(n, G, dk))), plain.unit(rng.normal(size=(n, G, dk)))
    v, g, beta = rng.normal(size=(n, H, dv)), rng.uniform(0.3, 1.0, size=(n, H, dk)), rng.uniform(0.1, 0.9, size=(n, H))
    if what == "forgets at once":
        g[:] = 0.0
    elif what == "never forgets":
        g[:] = 1.0
    elif what == "one key":
        k[:], g[:], beta[:] = k[0], 1.0, 0.999
    elif what == "two keys by turns":
        k[0::2], k[1::2] = k[0], -k[0]
        beta[:] = 0.99
    elif what == "far write":
        beta[:] = 0.0
        beta[5], g[:] = 1.0, 0.9995
        q[:] = 0.0
        q[-1] = k[5]
    elif what == "mixed channels":
        g[:, :, ::3], g[:, :, 1::3] = 0.0, 1.0
        g[::7] = 1e-30
    q, k, v, g, beta = (x.astype(np.float32).astype(np.float64) for x in (q, k, v, g, beta))
    own = np.arange(H) // (H // G)
    qkv = _f32(np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1))
    state = torch.zeros((1, H * dk * dv), device=DEV)
    o = kernels.delta_scan(qkv, _f32(g.reshape(n, -1)), _f32(beta), state, _i32([0, n]), _i32([0]), 1, n, G, H, dk, dv, chunked=chunked)
    want = plain.delta_rule(q[:, own], k[:, own], v, g, beta).reshape(n, -1)
    if what == "far write":
        assert np.abs(want[-1]).max() > 0.5
    err = np.abs(_np(o) - want).max()
    assert err <= 1e-5 * max(1.0, np.abs(want).max()), err


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dims", [(64, 64), (128, 128), (48, 48), (32, 32), (16, 24), (18, 10)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_capped_scores_and_learned_sinks_on_every_attention_kernel(dtype, dims, decode):
    """Hand-made queries, keys and values on scattered pages, scores far beyond the cap in both directions, sinks that weigh
    from nothing to almost everything, one and several slices of the key range: the tcgen05, the mma.sync and the CUDA-core
    kernel, each where it applies."""
    from llaisys_b200 import kernels
    from llaisys_b200.kernels import ops
    d, dv = dims
    H, G, L = 4, 2, 333
    rng = np.random.default_rng(d + dv)
    lens_before, n_new = ([L - 1, 70], [1, 1]) if decode else ([0, 100], [L, 90])
    T = sum(n_new)
    pages = sum(-(-(a + b) // 64) for a, b in zip(lens_before, n_new))
    perm = rng.permutation(pages + 3)
    kpool, vpool = (torch.full((pages + 3, G, 64, w), float("nan"), device=DEV, dtype=dtype) for w in (d, dv))
    table = np.zeros((2, 8), dtype=np.int64)
    keys, vals, at = [], [], 0
    for b in range(2):
        n = lens_before[b] + n_new[b]
        k, v = _bf16_exact(rng.normal(size=(n, G, d)) * 3), _bf16_exact(rng.normal(size=(n, G, dv)))
        for lp in range(-(-n // 64)):
            table[b, lp] = perm[at]
            m = min(64, n - lp * 64)
            kpool[perm[at], :, :m] = _f32(k[lp * 64:lp * 64 + m].transpose(1, 0, 2).copy()).to(dtype)
            vpool[perm[at], :, :m] = _f32(v[lp * 64:lp * 64 + m].transpose(1, 0, 2).copy()).to(dtype)
            at += 1
        keys.append(k)
        vals.append(v)
    q = _bf16_exact(rng.normal(size=(T, H, d)) * 3)
    proj = torch.zeros((T, H * d + G * (d + dv) + (-(H * d + G * (d + dv)) % 8)), device=DEV, dtype=dtype)
    proj[:, :H * d] = _f32(q.reshape(T, -1)).to(dtype)
    starts = np.concatenate([[0], np.cumsum(n_new)])
    sink, scale, cap = np.array([-4.0, 0.5, 3.0, 9.0]), 1.5 * d ** -0.5, 7.0
    extras = kernels.AttnExtras(value_dim=dv, sink_logits=_f32(sink), softcap=cap)
    args = (proj, H, G, d, kpool, vpool, _i32(table), 8, _i32(starts), _i32(lens_before), 2)
    outs = []
    if decode:
        outs = [kernels.attention_decode(*args, None, scale, n_splits=s, extras=extras) for s in (1, 2, 5)]
        if ops._mma_ok(proj, d) and d == dv:
            outs.append(kernels.attention_decode(*args, None, scale, n_splits=12, extras=extras))          # merged by a second kernel
    else:
        outs = [kernels.attention_prefill(*args, max(n_new), None, scale, all_from_cache=True, extras=extras)]
    for b in range(2):
        pos = lens_before[b] + np.arange(n_new[b])
        for h in range(H):
            qq = np.zeros((lens_before[b] + n_new[b], d))
            qq[pos] = q[starts[b]:starts[b + 1], h]
            raw = qq @ keys[b][:, h // 2].T * scale
            want = (plain.sink_softmax(plain.capped(raw, cap), sink[h]) @ vals[b][:, h // 2])[pos]
            for o in outs:
                got = _np(o)[starts[b]:starts[b + 1], h * dv:(h + 1) * dv]
                assert np.abs(got - want).max() <= (1e-5 if dtype == torch.float32 else 2e-2), (b, h)
    assert ops.tc_error(DEV) == 0


# ----------------------------------------------------------------------------- single layers
EDGE_CUTS = [[63, 2, 65, 1, 64], [2]]
LAYERS = {
    "attention": bh.attention(4, 2, 12, 20, softcap=5.0, rotation=bh.rot(8, 300.0, (4.0, 1.0, 3.0, 40))),
    "attention without cap and rotation": bh.attention(3, 1, 18, 10),
    "attention of one head": bh.attention(1, 1, 16, 16, softcap=50.0, rotation=bh.rot(16)),
    "delta": bh.delta(4, 2, 16, 12, 4, bh.dense(24, 0.9)),
    "delta with one tap": bh.delta(2, 2, 8, 20, 1),
    "delta with seven taps": bh.delta(3, 1, 10, 6, 7),
    "delta with twenty taps": bh.delta(2, 1, 64, 64, 20),
}


@pytest.mark.parametrize("name", sorted(LAYERS))
def test_one_layer_at_every_position(tmp_path, name):
    """280 positions whole, decoded one by one, and in portions that meet page and chunk borders from both sides."""
    cfg = bh.config(90, 32, [LAYERS[name]], embed_scale=4.0)
    folder = bh.make_folder(tmp_path, cfg, seed=len(name), gain=60.0)
    oracle = bh.Oracle(folder)
    toks = bh.random_requests(cfg, [280], seed=5)
    engine = build_engine(folder, torch.float32, max_tokens=320)
    compare_bz(run_whole(engine, toks), oracle, toks, torch.float32, cfg, "whole")
    compare_bz(run_tail_by_one(engine, toks, tail=270), oracle, toks, torch.float32, cfg, "decoded")
    for cuts in EDGE_CUTS:
        compare_bz(run_chunked(engine, toks, cuts), oracle, toks, torch.float32, cfg, f"portions {cuts}")


@pytest.mark.parametrize("layer", [bh.attention(4, 2, 64, 64, softcap=4.0, rotation=bh.rot(64, 1000.0, (4.0, 1.0, 4.0, 100))),
                                   bh.attention(2, 1, 128, 128, softcap=20.0, rotation=bh.rot(64, 1000.0)), bh.attention(3, 3, 48, 48, softcap=3.0),
                                   bh.attention(2, 1, 96, 96, rotation=bh.rot(96))], ids=["64", "128", "48", "96 uncapped"])
def test_attention_on_the_tensor_cores_against_the_cuda_cores(tmp_path, layer, monkeypatch):
    """bfloat16 prompts, portions and single tokens with the tensor-core attention kernels on and off: both against the plain
    implementation, and against each other row by row."""
    from llaisys_b200.kernels import ops
    cfg = bh.config(90, 64, [layer], embed_scale=4.0)
    folder = bh.make_folder(tmp_path, cfg, seed=3, gain=20.0)
    oracle = bh.Oracle(folder)
    toks = bh.random_requests(cfg, [300, 77], seed=5)
    got = {}
    for on in (True, False):
        monkeypatch.setattr(ops, "MMA_ATTENTION", on)
        monkeypatch.setattr(ops, "TC_ATTENTION", on)
        engine = build_engine(folder, torch.bfloat16, max_tokens=448, max_seqs=2)
        got[on] = (run_whole(engine, toks), run_chunked(engine, toks, [130, 70, 1000]), run_batches(engine, toks, [[0, 1]], [250, 30]))
        for g, what in zip(got[on], ("whole", "portions", "together")):
            compare_bz(g, oracle, toks, torch.bfloat16, cfg, f"{what}, tensor cores {on}")
    for a, b in zip(got[True], got[False]):
        for key, ref in b.items():
            rms = np.sqrt((ref.astype(np.float64) ** 2).mean())
            assert np.sqrt(((a[key] - ref).astype(np.float64) ** 2).mean()) <= 0.05 * rms + 1e-3, key


def _one_direction(cfg, special):
    """Attention: embeddings share one direction, the special token alone stands on the other side of it, and queries ask for
    that side, so its key gets the largest score of every later query.  Recurrent: only the special token has a step size
    (beta's row reads the direction), the state hardly decays, and every query is the special token's key."""
    def edit(t):
        D = cfg["width"]
        e = t["embed"].float()
        e *= 0.1 / e.std()
        e[:, 0] -= 1.0
        e[special] = 0.0
        e[special, 0] = 6.0
        t["embed"] = e.to(t["embed"].dtype)
        t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
        if cfg["layers"][0]["type"] == "attention":
            for n, rows, sign in (("l0.mix.q", cfg["layers"][0]["mixer"]["heads"], -3.0), ("l0.mix.k", cfg["layers"][0]["mixer"]["kv_heads"], 3.0)):
                m = torch.zeros((t[n].shape[0] // rows, D))
                m[0, 0] = sign
                t[n] = m.repeat(rows, 1).to(t[n].dtype)
        else:
            b = torch.zeros_like(t["l0.mix.b"].float())
            b[:, 0] = 10.0
            t["l0.mix.b"] = b.to(t["l0.mix.b"].dtype)
            t["l0.mix.A_log"] = torch.full_like(t["l0.mix.A_log"], -8.0)
            for n in ("l0.mix.q", "l0.mix.k"):
                m = torch.zeros_like(t[n].float())
                m[0::2, 0] = 3.0 if n.endswith("k") else -3.0
                t[n] = m.to(t[n].dtype)
            for n in ("l0.mix.q.conv", "l0.mix.k.conv", "l0.mix.v.conv"):
                c = torch.zeros_like(t[n].float())
                c[:, -1] = 1.0
                t[n] = c.to(t[n].dtype)
    return edit


@pytest.mark.parametrize("at", [0, 37, 63, 64, 65])
@pytest.mark.parametrize("layer", [bh.attention(2, 1, 16, 16, softcap=30.0), bh.delta(2, 1, 8, 12, 4)], ids=["attention", "delta"])
def test_one_far_token_that_decides(tmp_path, at, layer):
    """A token hundreds of positions back whose key dominates the softmax, or whose write is the state: whole, decoded, in
    portions.  The plain implementation itself moves by far more than the tolerance when that token is another one."""
    cfg = bh.config(64, 32, [layer])
    folder = bh.make_folder(tmp_path, cfg, seed=9, gain=1.0, edit=_one_direction(cfg, 63))
    oracle = bh.Oracle(folder)
    toks = np.random.default_rng(1).integers(0, 63, size=400).tolist()
    toks[at] = 63
    other = list(toks)
    other[at] = 5
    moved = np.abs(oracle.logits(toks)[-1] - oracle.logits(other)[-1]).max()
    assert moved > 100 * tolerance(torch.float32, bh.like_config(cfg), None), moved
    for dtype in DTYPES:
        engine = build_engine(folder, dtype, max_tokens=512)
        compare_bz(run_whole(engine, [toks]), oracle, [toks], dtype, cfg, f"far token {at} whole")
        compare_bz(run_tail_by_one(engine, [toks], tail=300), oracle, [toks], dtype, cfg, f"far token {at} decoded")
        compare_bz(run_chunked(engine, [toks], [at + 1, 2, 200, 64]), oracle, [toks], dtype, cfg, f"far token {at} portions")


def test_the_sequences_first_tokens_and_sizes_that_are_one(tmp_path):
    """Sequences of one to ten tokens (the convolution's window is not full, the state starts at zero, a softmax of one key
    and the sink), and a model of one head, one channel, one tap and one pass."""
    cfg = bh.CONFIGS["P"]
    folder = bh.make_folder(tmp_path / "p", cfg, seed=5, gain=40.0)
    reqs = bh.random_requests(cfg, [1, 2, 3, 4, 5, 8, 10], seed=1)
    engine = build_engine(folder, torch.float32, max_tokens=64 * 7, max_seqs=7)
    compare_bz(run_whole(engine, reqs), bh.Oracle(folder), reqs, torch.float32, cfg, "first tokens")
    compare_bz(run_batches(engine, reqs, [list(range(7))], [1] * 7), bh.Oracle(folder), reqs, torch.float32, cfg, "first tokens, decoded together")
    ones = bh.config(40, 16, [bh.delta(1, 1, 1, 1, 1, bh.dense(1, 1.0)), bh.attention(1, 1, 2, 1, softcap=1.0, rotation=bh.rot(2, 1.0), scale=1.0)],
                     loop=(0, 1, 1), logit_scale=1.0, embed_scale=1.0)
    folder = bh.make_folder(tmp_path / "ones", ones, seed=6, gain=4.0)
    reqs = bh.random_requests(ones, [70, 3], seed=2)
    engine = build_engine(folder, torch.float32, max_tokens=192)
    compare_bz(run_whole(engine, reqs), bh.Oracle(folder), reqs, torch.float32, ones, "ones whole")
    compare_bz(run_tail_by_one(engine, reqs, tail=60), bh.Oracle(folder), reqs, torch.float32, ones, "ones decoded")


def test_a_model_of_recurrent_layers_only(tmp_path):
    """A cache without page groups: long sequences hold nothing but their state rows, which are used again."""
    cfg = bh.config(70, 32, [bh.delta(2, 1, 16, 16, 4, bh.dense(16)), bh.delta(1, 1, 8, 24, 3)], loop=(0, 2, 2))
    for dtype in DTYPES:
        folder = bh.make_folder(tmp_path / str(dtype), cfg, seed=8, gain=1.0)
        oracle = bh.Oracle(folder)
        toks = bh.random_requests(cfg, [150, 20, 90], seed=9)
        engine = build_engine(folder, dtype, max_tokens=64, max_seqs=1)
        assert not engine.cache.group_keys
        for run in (run_whole(engine, toks), run_tail_by_one(engine, toks, tail=100), run_chunked(engine, toks, [63, 2, 65])):
            compare_bz(run, oracle, toks, dtype, cfg, "recurrent only")


# ----------------------------------------------------------------------------- whole models under every schedule
class Model:
    def __init__(self, name, tmp):
        self.name, self.tmp, self._made = name, tmp, {}

    def at(self, dtype):
        if dtype not in self._made:
            cfg = bh.CONFIGS[self.name]
            folder = bh.make_folder(self.tmp / str(dtype), cfg, seed=11, gain=bh.GAIN[dtype])
            self._made[dtype] = (cfg, folder, bh.Oracle(folder), bh.random_requests(cfg, [130, 1, 64, 65, 9, 201], seed=3))
        return self._made[dtype]


@pytest.fixture(scope="module", params=["P", "Q", "R"])
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp(f"bz{request.param}"))


def _rooms(requests):
    return sum(-(-len(r) // 64) * 64 for r in requests)


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_and_token_by_token(model, dtype):
    cfg, folder, oracle, requests = model.at(dtype)
    engine = build_engine(folder, dtype, max_tokens=max(_rooms([r]) for r in requests))
    compare_bz(run_whole(engine, requests), oracle, requests, dtype, cfg, f"{model.name} whole")
    compare_bz(run_tail_by_one(engine, requests, tail=10_000), oracle, requests, dtype, cfg, f"{model.name} token by token")
    compare_bz(run_tail_by_one(engine, requests, tail=32), oracle, requests, dtype, cfg, f"{model.name} tail")
    assert not engine.cache.live_slots


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_with_pages_slots_and_state_rows_used_again(model, dtype):
    cfg, folder, oracle, requests = model.at(dtype)
    n = len(requests)
    batches = [list(range(0, n, 2)), list(range(1, n, 2))]
    prompt_lens = [max(1, len(r) - (3 + 5 * i)) for i, r in enumerate(requests)]
    room = max(_rooms([requests[r] for r in b]) for b in batches)
    engine = build_engine(folder, dtype, max_tokens=room, max_seqs=len(batches[0]))
    compare_bz(run_batches(engine, requests, batches, prompt_lens), oracle, requests, dtype, cfg, f"{model.name} batches")
    assert not engine.cache.live_slots
    assert [p.available for p in engine.cache.book.pools] == engine.cache.group_pages
    compare_bz(run_batches(engine, requests, batches[::-1], prompt_lens), oracle, requests, dtype, cfg, f"{model.name} batches again")


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_mixed_steps(model, dtype):
    cfg, folder, oracle, _ = model.at(dtype)
    requests = bh.random_requests(cfg, [200, 300, 129, 9], seed=41)
    engine = build_engine(folder, dtype, max_tokens=320)
    for cuts in ([70, 60, 1000], [63, 1, 64, 65, 2, 1000], [2, 200, 1000], [64], [2]):
        reqs = requests if cuts != [2] else requests[2:]
        compare_bz(run_chunked(engine, reqs, cuts), oracle, reqs, dtype, cfg, f"{model.name} portions {cuts}")
    requests = bh.random_requests(cfg, [120, 100, 210, 33], seed=43)
    plans = [[50, 1, 1, 1, 40, 1, 0, 1], [0, 0, 90], [70, 60, 0, 40, 1, 1, 30], [1, 1, 1]]
    engine = build_engine(folder, dtype, max_tokens=_rooms(requests), max_seqs=4)
    for turn in range(2):
        compare_bz(run_mixed(engine, requests, plans), oracle, requests, dtype, cfg, f"{model.name} mixed steps, turn {turn}")
        assert not engine.cache.live_slots
        requests, plans = requests[::-1], plans[::-1]


def test_bfloat16_does_not_depend_on_how_the_steps_are_cut(model):
    """bfloat16 logits of whole prompts (recurrence in chunks on the tensor cores), of portions, of unequal batches and of
    single tokens (recurrence token by token) agree with one another far more closely than either with exact arithmetic
    where a vector of few elements is normed: a stale state row or a page of another sequence moves every later row."""
    cfg, folder, _, _ = model.at(torch.bfloat16)
    requests = bh.random_requests(cfg, [150, 70, 9], seed=2)
    engine = build_engine(folder, torch.bfloat16, max_tokens=_rooms(requests), max_seqs=3)
    whole = run_whole(engine, requests)
    for what, other in (("portions", run_chunked(engine, requests, [63, 2, 65])), ("together", run_batches(engine, requests, [[0, 1, 2]], [100, 64, 1])),
                        ("decoded", run_tail_by_one(engine, requests, tail=40))):
        off = 0
        for key, ref in whole.items():
            rms = np.sqrt((ref.astype(np.float64) ** 2).mean())
            d = np.sqrt(((other[key] - ref).astype(np.float64) ** 2).mean())
            off += d > 0.05 * rms + 1e-3
        assert off <= max(2, len(whole) // 25), (what, off, len(whole))


def test_long_decoding_through_captured_steps(tmp_path):
    """Hundreds of single-token steps from a short prompt: pages fill and new ones are taken, the state and the convolutions'
    inputs are carried through every step, and the steps are replayed from a captured graph."""
    for dtype in DTYPES:
        cfg = bh.CONFIGS["P"]
        folder = bh.make_folder(tmp_path / str(dtype), cfg, seed=21, gain=bh.GAIN[dtype])
        oracle = bh.Oracle(folder)
        requests = bh.random_requests(cfg, [330, 290], seed=6)
        engine = build_engine(folder, dtype, max_tokens=_rooms(requests), max_seqs=2)
        assert engine.use_graphs
        compare_bz(run_batches(engine, requests, [[0, 1]], [4, 1]), oracle, requests, dtype, cfg, "long decoding")
        assert engine.graph_replays > 250


# ----------------------------------------------------------------------------- entry points
def _greedy(oracle, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(oracle.logits(seq)[-1])))
    return seq[len(prompt):]


def test_greedy_generation_through_the_entry_point_and_scheduler(tmp_path):
    from llaisys_b200.models import CausalLM, DeviceType
    cfg = bh.CONFIGS["P"]
    folder = bh.make_folder(tmp_path, cfg, seed=31, gain=40.0)
    oracle = bh.Oracle(folder)
    model = CausalLM(folder, DeviceType.NVIDIA, dtype="float32", max_tokens=64 * 4)
    prompts = bh.random_requests(cfg, [5, 9, 2, 70, 1, 17], seed=3)
    # four rooms of 64 tokens for six requests: two batches at least; slots, pages and state rows are used again
    outs = model.generate_batch(prompts, max_new_tokens=12, top_k=1, stop_ids=[])
    for p, new in zip(prompts, outs):
        assert new == _greedy(oracle, p, 12)
    assert model.generate(prompts[0], max_new_tokens=12) == prompts[0] + outs[0]
    assert not model.engine.cache.live_slots


def test_command_line(tmp_path):
    """python -m llaisys_b200.cli on a model folder of this design and on a configuration with random weights; --test
    compares the engine's tokens with those of the package's CPU model."""
    import os
    import sys
    env = dict(os.environ, PYTHONPATH=str(ROOT))
    folder = bh.make_folder(tmp_path / "m", bh.CONFIGS["P"], seed=17, gain=40.0)
    oracle = bh.Oracle(folder)
    (tmp_path / "batch.txt").write_text("5,17,3,200,7,7,7,7,7\n[9, 8]\n1\n")
    out = subprocess.run([sys.executable, "-m", "llaisys_b200.cli", "--model", str(folder), "--batch-file", str(tmp_path / "batch.txt"),
                          "--max_steps", "6", "--dtype", "float32", "--test"], env=env, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert out.stdout.count("Tokens:") == 3 and "Test passed" in out.stdout
    want = [5, 17, 3, 200, 7, 7, 7, 7, 7] + _greedy(oracle, [5, 17, 3, 200, 7, 7, 7, 7, 7], 6)
    assert str(want) in out.stdout or ", ".join(map(str, want)) in out.stdout, out.stdout[-1500:]
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(bh.CONFIGS["Q"]))
    out = subprocess.run([sys.executable, "-m", "llaisys_b200.cli", "--random-weights", str(cfg), "--seed", "3", "--tokens", "1,2,3",
                          "--max_steps", "4", "--dtype", "float32", "--test"], env=env, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert "Tokens:" in out.stdout and "Test passed" in out.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_of_a_trace(tmp_path, dtype):
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    cfg = bh.CONFIGS["P"]
    folder = bh.make_folder(tmp_path / "m", cfg, seed=13, gain=bh.GAIN[td])
    requests = bh.random_requests(cfg, [1, 7, 90, 20], seed=8)
    lines, rows = [], []
    lines.append({"step": 0, "entries": [{"id": "a", "tokens": requests[0], "want": [0]},
                                         {"id": "c", "tokens": requests[2][:60], "want": list(range(60))}], "end": ["a"]})
    rows.append((0, [(0, 0)] + [(2, p) for p in range(60)]))
    for p in range(60, 90):
        lines.append({"step": p, "entries": [{"id": "c", "tokens": [requests[2][p]], "want": [0]}], "end": ["c"] if p == 89 else []})
        rows.append((p, [(2, p)]))
    lines.append({"step": 500, "entries": [], "end": []})
    lines.append({"step": 501, "entries": [{"id": "b", "tokens": requests[1], "want": list(range(7))},
                                           {"id": "d", "tokens": requests[3], "want": [19]}], "end": ["b", "d"]})
    rows.append((501, [(1, p) for p in range(7)] + [(3, 19)]))
    out_dir = tmp_path / "out"
    proc = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out_dir),
                           "--max-tokens", "128"], input="\n".join(json.dumps(l) for l in lines) + "\n", capture_output=True,
                          text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [int(l.split()[1]) for l in proc.stdout.splitlines() if l.startswith("done ")] == [l["step"] for l in lines]
    oracle = bh.Oracle(folder)
    for step, keys in rows:
        data = np.frombuffer((out_dir / f"{step}.f32").read_bytes(), dtype="<f4").reshape(len(keys), cfg["vocab"])
        for i, (r, p) in enumerate(keys):
            ref = oracle.logits(requests[r])
            assert np.abs(data[i] - ref[p]).max() <= tolerance(td, bh.like_config(cfg), ref) * (1 if dtype == "float32" else 8), (step, r, p)

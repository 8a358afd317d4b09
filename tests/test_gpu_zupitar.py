"""The Zupitar design on the GPU against its plain implementation: every mechanism alone, then single layers at the places
where a fault would hide (page and chunk borders, a key far back, the first tokens, long memory), then whole models under every
way of cutting requests into steps, then generation and replay through the entry points."""
import json
import subprocess
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_zupitar as plain
import zupitar_helpers as zh
from helpers import build_engine, run_batches, run_chunked, run_mixed, run_tail_by_one, run_whole, tolerance
from zupitar_helpers import compare

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


def _env(dtype):
    from llaisys_b200.parts import BuildEnv
    return BuildEnv(dtype, torch.device(DEV))


def _ctx(slots, before, new):
    starts = np.concatenate([[0], np.cumsum(new)])
    pos = np.concatenate([np.arange(b, b + n) for b, n in zip(before, new)])
    return SimpleNamespace(seq_start=_i32(starts), seq_slot=_i32(slots), seq_len_before=_i32(before), tok_pos=_i32(pos), n_seqs=len(new),
                           max_new=int(max(new)), n_new=list(new), err=torch.zeros(1, dtype=torch.int32, device=DEV))


CUTS = [(1000,), (1,), (2, 1, 3, 7, 1, 1, 40), (16, 15, 17, 1, 1000)]
CUT_NAMES = ["whole", "single", "small", "portions"]


def _portions(lens, cuts):
    """[(live sequences, tokens before, new tokens)] of sequences fed together, each by its own slightly different portions."""
    at, i, out = [0] * len(lens), 0, []
    while any(a < n for a, n in zip(at, lens)):
        n = cuts[min(i, len(cuts) - 1)]
        i += 1
        live = [b for b in range(len(lens)) if at[b] < lens[b]]
        new = [min(n + (b if n > 1 else 0), lens[b] - at[b]) for b in live]
        out.append((live, [at[b] for b in live], new))
        for b, m in zip(live, new):
            at[b] += m
    return out


# ----------------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("cuts", CUTS, ids=CUT_NAMES)
@pytest.mark.parametrize("C, taps", [(64, 4), (7, 4), (130, 1), (33, 3), (96, 6), (40, 13)])
def test_short_convolution_with_inputs_carried_in_slots(C, taps, cuts):
    """Three sequences whose portions share steps; their carried inputs lie in state rows in another order than the batch; inputs
    are a slice of a wider matrix; both input types, with and without bias and activation."""
    from llaisys_b200 import kernels
    lens, slots = [40, 9, 23], [2, 0, 3]
    rng = np.random.default_rng(C + taps)
    w, bias = rng.uniform(-1, 1, size=(C, taps)), rng.normal(size=C)
    x = [_bf16_exact(rng.normal(size=(n, C))) for n in lens]
    wd = _f32(w.T.copy()).contiguous()
    for xt, ot, act in ((torch.float32, torch.float32, "silu"), (torch.bfloat16, torch.bfloat16, None), (torch.float32, torch.bfloat16, "silu")):
        state = torch.full((4, max(1, (taps - 1) * C)), 7.0, device=DEV)
        for s in slots:
            state[s].zero_()
        got = [[] for _ in lens]
        for live, before, new in _portions(lens, cuts):
            wide = torch.zeros((sum(new), C + 8 + -C % 4), device=DEV, dtype=xt)
            wide[:, 4:4 + C] = _f32(np.concatenate([x[b][a:a + m] for b, a, m in zip(live, before, new)])).to(xt)
            y = kernels.short_conv(wide[:, 4:4 + C], wd, _f32(bias) if act else None, state if taps > 1 else None, _ctx([slots[b] for b in live], before, new),
                                   act=act, out_dtype=ot)
            o = 0
            for b, m in zip(live, new):
                got[b].append(y[o:o + m])
                o += m
        assert (state[1] == 7.0).all()
        for b in range(3):
            want = plain.short_conv(x[b], w, bias if act else None)
            _close(torch.cat(got[b]), plain.silu(want) if act else want, 2e-6 if ot == torch.float32 else 4e-3, (b, xt, ot))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", CUTS, ids=CUT_NAMES)
@pytest.mark.parametrize("H, G, d, dims, taps", [(4, 2, 16, 12, 4), (3, 1, 7, 4, 3), (2, 2, 18, 0, 4), (2, 1, 64, 64, 4), (6, 2, 24, 8, 1), (1, 1, 9, 2, 12)])
def test_convolved_heads_their_values_rotation_and_cache_rows(H, G, d, dims, taps, cuts, dtype):
    """Queries and keys rotated by position, values that are the keys before the rotation times a constant, and the rows of the
    paged cache on scattered pages, from portions that cross page borders."""
    from llaisys_b200 import kernels
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import build_part
    lens, slots, mult = [150, 9, 70], [1, 2, 0], -1.5
    if cuts == (1,):
        lens = [66, 3, 5]
    rng = np.random.default_rng(H + d)
    C = (H + G) * d
    w = rng.uniform(-1, 1, size=(C, taps))
    x = [_bf16_exact(rng.normal(size=(n, C))) for n in lens]
    r = {"dims": dims, "base": 300.0, "scaling": {"factor": 2.5}}
    tables = None
    if dims:
        part = build_part("position", PartSpec("rope_leading", {"head_dim": d, "dims": dims, "base": 300.0, "factor": 2.5}), _env(dtype))
        tables = part.pair_tables(256)
    perm = rng.permutation(9)
    kpool, vpool = (torch.full((9, G, 64, d), 5.0, device=DEV, dtype=dtype) for _ in range(2))
    table = np.stack([perm[3 * b:3 * b + 3] for b in range(3)])
    state = torch.zeros((3, max(1, (taps - 1) * C)), device=DEV)
    wd = _f32(w.T.copy()).contiguous()
    got = [[] for _ in lens]
    for live, before, new in _portions(lens, cuts):
        ctx = _ctx([slots[b] for b in live], before, new)
        append = dict(seq_len_before=ctx.seq_len_before, kpool=kpool, vpool=vpool, page_table=_i32(table[live]), ring=3, pinned=0)
        xs = _f32(np.concatenate([x[b][a:a + m] for b, a, m in zip(live, before, new)])).to(dtype)
        out = kernels.conv_heads(xs, H, G, d, wd, state if taps > 1 else None, ctx, tables, mult, append)
        assert int(ctx.err.item()) == 0
        o = 0
        for b, m in zip(live, new):
            got[b].append(out[o:o + m])
            o += m
    tol = 5e-6 if dtype == torch.float32 else 8e-3
    for b, n in enumerate(lens):
        y = plain.short_conv(x[b], w)
        q, k = y[:, :H * d].reshape(n, H, d), y[:, H * d:].reshape(n, G, d)
        v, q, k = k * mult, plain.rotate(q, np.arange(n), r), plain.rotate(k, np.arange(n), r)
        _close(torch.cat(got[b]), np.concatenate([t.reshape(n, -1) for t in (q, k, v)], 1), tol, "packed")
        for pool, want in ((kpool, k), (vpool, v)):
            rows = torch.stack([pool[int(table[b, p // 64]), :, p % 64] for p in range(n)])
            _close(rows, want, tol, "cache")
    used = {(int(table[b, p // 64]), p % 64) for b, n in enumerate(lens) for p in range(n)}
    for page in range(9):
        for row in range(64):
            if (page, row) not in used:
                assert (kpool[page, :, row] == 5.0).all() and (vpool[page, :, row] == 5.0).all()


def _ssd_case(H, P, N, G, lens, seed, rates=(-4.0, 1.0), bf16=True):
    rng = np.random.default_rng(seed)
    C = H * P + 2 * G * N
    exact = _bf16_exact if bf16 else (lambda a: a.astype(np.float32).astype(np.float64))
    return dict(xbc=[exact(rng.normal(size=(n, C))) for n in lens], dt=[rng.normal(size=(n, H)) * 2 for n in lens], bias=rng.uniform(-3, 1, size=H),
                a_log=rng.uniform(*rates, size=H), skip=rng.uniform(-1, 1, size=H))


def _ssd_want(case, b, H, P, N, G):
    x, n = case["xbc"][b], len(case["xbc"][b])
    own = np.arange(H) // (H // G)
    B, C = (x[:, H * P + i * G * N:H * P + (i + 1) * G * N].reshape(n, G, N)[:, own] for i in (0, 1))
    return plain.state_space(x[:, :H * P].reshape(n, H, P), B, C, plain.softplus(case["dt"][b] + case["bias"]), -np.exp(case["a_log"]),
                             case["skip"]).reshape(n, -1)


SSD_SHAPES = [(4, 8, 16, 2), (6, 16, 24, 3), (3, 5, 6, 3), (2, 9, 13, 1), (3, 7, 33, 1), (1, 1, 1, 1), (2, 64, 128, 1), (1, 72, 136, 1), (2, 8, 256, 2),
              (1, 130, 40, 1), (4, 32, 64, 4), (2, 66, 17, 2)]


def _run_ssd(case, lens, slots, cuts, H, P, N, G, dtype, chunked):
    """chunked: None, or the tokens from which a step runs in chunks."""
    from llaisys_b200 import kernels
    state = torch.full((4, H * N * P), 7.0, device=DEV)
    for s in slots:
        state[s].zero_()
    got = [[] for _ in lens]
    vecs = [_f32(case[k]) for k in ("bias", "a_log", "skip")]
    for live, before, new in _portions(lens, cuts):
        ctx = _ctx([slots[b] for b in live], before, new)
        cat = lambda k: _f32(np.concatenate([case[k][b][a:a + m] for b, a, m in zip(live, before, new)]))
        dt = torch.zeros((sum(new), H + 3), device=DEV)
        dt[:, 2:2 + H] = cat("dt")
        y = kernels.ssd_scan(cat("xbc").to(dtype), dt[:, 2:2 + H], *vecs, state, ctx.seq_start, ctx.seq_slot, ctx.n_seqs, ctx.max_new, H, P, N, G,
                             chunked=chunked is not None and max(new) >= chunked)
        o = 0
        for b, m in zip(live, new):
            got[b].append(y[o:o + m])
            o += m
    assert (state[1] == 7.0).all()
    return [torch.cat(g) for g in got], state


@pytest.mark.parametrize("cuts", CUTS, ids=CUT_NAMES)
@pytest.mark.parametrize("shape", SSD_SHAPES, ids=[str(s) for s in SSD_SHAPES])
def test_state_space_recurrence_token_by_token(shape, cuts):
    lens, slots = [40, 9, 23], [2, 0, 3]
    for dtype in DTYPES:
        case = _ssd_case(*shape, lens, seed=sum(shape), bf16=dtype == torch.bfloat16)
        got, _ = _run_ssd(case, lens, slots, cuts, *shape, dtype, None)
        for b in range(3):
            _close(got[b], _ssd_want(case, b, *shape), 5e-6, (dtype, b))


@pytest.mark.parametrize("cuts", [(1000,), (64, 1, 63, 65, 1000), (2, 130, 1, 1, 40)], ids=["whole", "borders", "mixed"])
@pytest.mark.parametrize("shape", SSD_SHAPES, ids=[str(s) for s in SSD_SHAPES])
def test_state_space_recurrence_in_chunks(shape, cuts):
    """Chunks on the tensor cores against the plain recurrence, far closer than 16-bit operands would give: portions that end just
    before, at and just behind a chunk's border, short sequences beside long ones, and steps token by token in between; the states
    left behind agree with those of the token-by-token kernel."""
    lens, slots = [200, 1, 129], [2, 0, 3]
    case = _ssd_case(*shape, lens, seed=1 + sum(shape))
    got, state = _run_ssd(case, lens, slots, cuts, *shape, torch.bfloat16, 2)
    for b in range(3):
        want = _ssd_want(case, b, *shape)
        assert np.abs(_np(got[b]) - want).max() <= 1e-4 * max(1.0, np.abs(want).max()), b
    _, ref = _run_ssd(case, lens, slots, (1000,), *shape, torch.bfloat16, None)
    assert (state - ref).abs().max() <= 1e-4 * max(1.0, float(ref[slots].abs().max()))


@pytest.mark.parametrize("what", ["kept", "forgotten at once", "one write far back", "steps of zero", "large steps"])
@pytest.mark.parametrize("chunked", [False, True])
def test_state_space_recurrence_at_its_extremes(what, chunked):
    H, P, N, G = 2, 16, 32, 1
    n = 300
    case = _ssd_case(H, P, N, G, [n], seed=5)
    if what == "kept":
        case["a_log"][:] = -12.0
    if what == "forgotten at once":
        case["a_log"][:] = 5.0
    if what == "one write far back":                       # only token 3 writes; the state then hardly decays
        case["a_log"][:] = -9.0
        case["dt"][0][:] = -60.0
        case["dt"][0][3] = 3.0
    if what == "steps of zero":
        case["dt"][0][::3] = -80.0
    if what == "large steps":
        case["dt"][0][::50] = 40.0
    got, _ = _run_ssd(case, [n], [2], (1000,), H, P, N, G, torch.bfloat16, 2 if chunked else None)
    want = _ssd_want(case, 0, H, P, N, G)
    if what == "one write far back":
        assert np.abs(want[-1] - (case["skip"][:, None] * case["xbc"][0][-1, :H * P].reshape(H, P)).reshape(-1)).max() > 1.0
    _close(got[0], want, 1e-4 if chunked else 1e-5, what)


@pytest.mark.parametrize("groups, size", [(1, 64), (3, 7), (2, 512), (1, 900), (4, 1536), (2, 1), (5, 33)])
@pytest.mark.parametrize("T", [1, 5, 40])
def test_gate_and_norm_in_parts(groups, size, T):
    from llaisys_b200 import kernels
    rng = np.random.default_rng(groups + size)
    C = groups * size
    y, z, w = rng.normal(size=(T, C)) * rng.uniform(0.1, 9, size=(T, 1)), _bf16_exact(rng.normal(size=(T, C)) * 2), rng.uniform(0.5, 1.5, size=C)
    want = plain.gated_group_norm(y, z, w, groups, 1e-5)
    for zt in DTYPES:
        wide = torch.zeros((T, C + 8 + -C % 4), device=DEV, dtype=zt)
        wide[:, :C] = _f32(z).to(zt)
        _close(kernels.gated_group_norm(_f32(y), wide[:, :C], _f32(w), groups, 1e-5, torch.float32), want, 1e-5, "float32")
        _close(kernels.gated_group_norm(_f32(y), wide[:, :C], _f32(w), groups, 1e-5, torch.bfloat16), want, 6e-3, "bfloat16")


ROUTERS = [(7, 2, 3, (3, 2)), (6, 0, 3, (2, 1)), (3, 2, 2, None), (4, 4, 4, (4, 2)), (5, 0, 1, None), (1, 1, 1, None), (40, 8, 6, (8, 3)), (2, 6, 3, (4, 2))]


@pytest.mark.parametrize("T", [1, 9, 300])
@pytest.mark.parametrize("experts, identity, top, groups", ROUTERS)
def test_softmax_router_with_groups_and_identity_experts(experts, identity, top, groups, T):
    """Choice and weights from logits made by an exact product; corrections that make choice scores negative and change the
    choice; the identity experts' weights summed."""
    from llaisys_b200 import kernels
    E = experts + identity
    rng = np.random.default_rng(E + top)
    D = E + (-E % 8)
    w, x = np.eye(E, D), _bf16_exact(rng.normal(size=(T, D)) * 2)
    bias = rng.uniform(-0.5, 0.2, size=E)
    r = {"experts": experts, "identity": identity, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    want_idx, want_w = plain.route(x @ w.T, bias.astype(np.float32).astype(np.float64), r)
    out = kernels.moe_route(_f32(x), _f32(w), _f32(bias), top, 1.0, gate="softmax", groups=groups, group_max=True, identity=identity)
    assert np.array_equal(out[0].cpu().numpy(), want_idx)
    _close(out[1], want_w, 2e-6)
    if identity:
        _close(out[2], np.where(want_idx >= experts, want_w, 0.0).sum(axis=1), 2e-6)
    assert (want_idx != plain.route(x @ w.T, np.zeros(E), r)[0]).any() or T < 300 or E <= 2, "the correction decides nothing"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 5, 70, 300])
@pytest.mark.parametrize("experts, identity, top, groups", ROUTERS)
def test_gated_experts_beside_identity_experts(experts, identity, top, groups, T, dtype):
    """The part against the plain mixture where both sides make the same choice: returned, and added to a stream; also steps in which
    every token, or none, uses an identity expert only."""
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import build_part
    D, ff = 64, 40
    rng = np.random.default_rng(experts + T)
    E = experts + identity
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    for tilt in ((0.0, 1000.0, -1000.0) if identity >= top and T == 5 and not groups else (0.0,)):
        w = {"router": np.round(rng.normal(size=(E, D)) * 4) / 8, "correction": _bf16_exact(rng.uniform(-0.5, 0.2, size=E))}
        w["correction"][experts:] += tilt
        for e in range(experts):
            w.update({f"e{e}.gate": _bf16_exact(rng.normal(size=(ff, D)) * 0.3), f"e{e}.up": _bf16_exact(rng.normal(size=(ff, D)) * 0.3),
                      f"e{e}.down": _bf16_exact(rng.normal(size=(D, ff)) * 0.3)})
        x = _bf16_exact(rng.normal(size=(T, D)))
        part = build_part("ffn", PartSpec("routed_experts", {
            "hidden_size": D, "experts": experts, "top": top, "identity": identity, "expert_ff": ff, "gate": "softmax", "act": "silu",
            "groups": router.get("groups"), "group_score": "max", "use_bias": True}), _env(dtype))
        part.load({k: _f32(v).to(dtype) if k != "correction" else _f32(v) for k, v in w.items()})
        want = plain.moe(x, w, {"router": router, "expert": {"ff": ff}})
        if tilt and identity >= top:
            used = plain.route(x @ w["router"].T, w["correction"], router)[0]
            assert (used >= experts).all() if tilt > 0 else (used >= experts).sum() == max(0, top - experts) * T
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        _close(part.forward(_f32(x).to(dtype), None), want, tol, "returned")
        stream = torch.full((T, D), 3.0, device=DEV)
        assert part.forward_into(_f32(x).to(dtype), None, stream)
        _close(stream - 3.0, want, tol, "into the stream")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 20, 40, 100, 300])
def test_relu_gated_feed_forward(dtype, T):
    """Every product kernel that ends in the gated activation, with gates of both signs, zeros and values far from zero."""
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.parts import build_part
    for D, F in ((64, 96), (136, 200), (44, 30)):
        rng = np.random.default_rng(T + D)
        w = {"gate": _bf16_exact(rng.normal(size=(F, D)) * 0.3), "up": _bf16_exact(rng.normal(size=(F, D)) * 0.3), "down": _bf16_exact(rng.normal(size=(D, F)) * 0.3)}
        w["gate"][0] = 0.0
        w["gate"][1] *= 1e4
        w["down"][:, 1] *= 1e-4
        h = _bf16_exact(rng.normal(size=(T, D)))
        part = build_part("ffn", PartSpec("gated_mlp", {"hidden_size": D, "intermediate_size": F, "act": "relu", "names": {k: k for k in w}}), _env(dtype))
        part.load({k: _f32(v).to(dtype) for k, v in w.items()})
        want, tol = plain.dense(h, w), 2e-5 if dtype == torch.float32 else 2e-2
        _close(part.forward(_f32(h).to(dtype), None), want, tol, "returned")
        stream = torch.full((T, D), 3.0, device=DEV)
        if part.forward_into(_f32(h).to(dtype), None, stream):
            _close(stream - 3.0, want, tol, "into the stream")


def test_cap_of_the_logits_and_output_norms_of_every_width():
    from llaisys_b200 import kernels
    rng = np.random.default_rng(0)
    z = rng.normal(size=(5, 77)) * 30
    _close(kernels.softcap_(_f32(z), 7.0), plain.capped(z, 7.0), 1e-6)
    for H in (4, 44, 50, 1000, 1028, 2048, 3000, 4096, 8192, 8196):
        x, d, w, v = rng.normal(size=(3, H)), rng.normal(size=(3, H)) * 4, rng.uniform(0.5, 1.5, size=H), rng.uniform(0.5, 1.5, size=H)
        new = x + 0.5 * plain.rms(d, 1e-5) * w
        for wt in DTYPES:
            wd, vd = _f32(w).to(wt), _f32(v).to(wt)
            for ot in DTYPES:
                xd = _f32(x)
                out = kernels.scaled_norm_add(xd, _f32(d), wd, 0.5, vd, 1e-5, 0.0, ot)
                tol = 2e-5 if wt == torch.float32 else 4e-3
                _close(xd, new, tol, H)
                _close(out, plain.rms(new, 1e-5) * v, tol if ot == torch.float32 else 8e-3, H)
            xd = _f32(x)
            _close(kernels.scaled_norm_add(xd, None, None, 1.0, vd, 1e-5, 0.0, torch.float32), plain.rms(x, 1e-5) * v, 2e-5 if wt == torch.float32 else 4e-3, H)
            assert kernels.scaled_norm_add(xd, _f32(d), wd, 0.5, None, 1e-5, 0.0) is None
            _close(xd, new, 2e-5 if wt == torch.float32 else 4e-3, H)


# ----------------------------------------------------------------------------- single layers
EDGE_CUTS = [[63, 2, 65, 1, 64], [2]]
LAYERS = {
    "parallel": zh.parallel((4, 2, 12, 4, zh.rot(8, 300.0, 3.0)), (2, 8, 16, 1, 4, 2), (0.7, 1.4)),
    "parallel without convolution and rotation": zh.parallel((3, 1, 18, None, None), (1, 6, 5, 1, 3, 1)),
    "parallel without the state space": zh.parallel((2, 1, 16, 3, zh.rot(16, 50.0)), (1, 4, 4, 1, 2, 1), (1.0, 0.0)),
    "mamba2": zh.mamba2(4, 12, 20, 2, 4, 2, mlp=zh.dense(24)),
    "mamba2 with one tap": zh.mamba2(2, 8, 16, 2, 1, 1),
    "mamba2 with twenty taps": zh.mamba2(1, 64, 64, 1, 20, 1, mlp=zh.moe(3, 2, 16, 1)),
}


@pytest.mark.parametrize("name", sorted(LAYERS))
def test_one_layer_at_every_position(tmp_path, name):
    """280 positions whole, decoded one by one, and in portions that meet page and chunk borders from both sides."""
    cfg = zh.config(90, 32, [LAYERS[name]])
    folder = zh.make_folder(tmp_path, cfg, seed=len(name), gain=60.0)
    oracle = zh.Oracle(folder)
    toks = zh.random_requests(cfg, [280], seed=5)
    engine = build_engine(folder, torch.float32, max_tokens=320)
    compare(run_whole(engine, toks), oracle, toks, torch.float32, cfg, "whole")
    compare(run_tail_by_one(engine, toks, tail=270), oracle, toks, torch.float32, cfg, "decoded")
    for cuts in EDGE_CUTS:
        compare(run_chunked(engine, toks, cuts), oracle, toks, torch.float32, cfg, f"portions {cuts}")


@pytest.mark.parametrize("dim, dims", [(64, 64), (128, 64), (48, 0), (96, 96)])
def test_attention_on_the_tensor_cores_against_the_cuda_cores(tmp_path, dim, dims, monkeypatch):
    """bfloat16 prompts, portions and single tokens with the tensor-core attention kernels on and off: both against the plain
    implementation, and against each other row by row."""
    from llaisys_b200.kernels import ops
    cfg = zh.config(90, 64, [zh.parallel((4, 2, dim, 4, zh.rot(dims, 1000.0, 2.0) if dims else None), (1, 16, 16, 1, 4, 1), (1.2, 0.3))])
    folder = zh.make_folder(tmp_path, cfg, seed=3, gain=20.0)
    oracle = zh.Oracle(folder)
    toks = zh.random_requests(cfg, [300, 77], seed=5)
    got = {}
    for on in (True, False):
        monkeypatch.setattr(ops, "MMA_ATTENTION", on)
        monkeypatch.setattr(ops, "TC_ATTENTION", on)
        engine = build_engine(folder, torch.bfloat16, max_tokens=448, max_seqs=2)
        got[on] = (run_whole(engine, toks), run_chunked(engine, toks, [130, 70, 1000]), run_batches(engine, toks, [[0, 1]], [250, 30]))
        for g, what in zip(got[on], ("whole", "portions", "together")):
            compare(g, oracle, toks, torch.bfloat16, cfg, f"{what}, tensor cores {on}")
    for a, b in zip(got[True], got[False]):
        for key, ref in b.items():
            rms = np.sqrt((ref.astype(np.float64) ** 2).mean())
            assert np.sqrt(((a[key] - ref).astype(np.float64) ** 2).mean()) <= 0.05 * rms + 1e-3, key


def _one_direction(cfg, special):
    """Embeddings share one direction; the special token alone stands on the other side of it.  Attention (right scale 0): queries ask
    for that side, so its key gets the largest score of every later query.  State space: only the special token has a step size (dt
    reads the direction), the state hardly decays, and every token reads what it wrote."""
    def edit(t):
        D = cfg["width"]
        e = t["embed"].float()
        e *= 0.1 / e.std()
        e[:, 0] -= 1.0
        e[special] = 0.0
        e[special, 0] = 6.0
        t["embed"] = e.to(t["embed"].dtype)
        t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
        layer = cfg["layers"][0]
        if layer["type"] == "parallel":
            m = layer["mixer"]["left"]
            for n, rows, sign in (("q", m["heads"], -3.0), ("k", m["kv_heads"], 3.0)):
                w = torch.from_numpy(np.random.default_rng(1).normal(size=(m["dim"], D)) * 0.05).float()
                w[:, 0] = torch.where(torch.arange(m["dim"]) == 0, sign, 0.5)
                t[f"l0.mix.left.{n}"] = w.repeat(rows, 1).to(t["embed"].dtype)
                c = torch.zeros((rows * m["dim"], m["conv"]))
                c[:, -1] = 1.0
                t[f"l0.mix.left.{n}.conv"] = c.to(t["embed"].dtype)
            return
        m = layer["mixer"]
        w = t["l0.mix.in"].float()
        w[-m["heads"]:] = 0.0
        w[-m["heads"]:, 0] = 20.0                          # dt: large and positive for the special token, far below zero for others
        # what is written and what is asked for are fixed (a read-out near zero would leave its direction to rounding)
        inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
        w[2 * inner:2 * inner + 2 * gn] = 0.0
        w[2 * inner:2 * inner + gn, 0] = torch.linspace(0.5, 1.0, gn)
        w[2 * inner + gn:2 * inner + 2 * gn, 0] = -torch.linspace(1.0, 0.5, gn)
        conv, bias = t["l0.mix.conv"].float(), t["l0.mix.conv.b"].float()
        conv[inner:, :-1], conv[inner:, -1], bias[inner:] = 0.0, 1.0, 0.0
        t["l0.mix.conv"], t["l0.mix.conv.b"] = conv.to(t["embed"].dtype), bias.to(t["embed"].dtype)
        t["l0.mix.in"] = w.to(t["embed"].dtype)
        t["l0.mix.A_log"] = torch.full_like(t["l0.mix.A_log"], -9.0)
        t["l0.mix.dt_bias"] = torch.full_like(t["l0.mix.dt_bias"], -3.0)
        t["l0.mix.D"] = torch.zeros_like(t["l0.mix.D"])
    return edit


@pytest.mark.parametrize("at", [0, 37, 63, 64, 65])
@pytest.mark.parametrize("layer", [zh.parallel((2, 1, 16, 4, None), (1, 4, 4, 1, 2, 1), (1.0, 0.0)), zh.mamba2(2, 8, 12, 1, 4, 1)], ids=["attention", "state space"])
def test_one_far_token_that_decides(tmp_path, at, layer):
    """A token hundreds of positions back whose key dominates the softmax, or whose write is the state: whole, decoded, in
    portions.  The plain implementation itself moves by far more than the tolerance when that token is another one."""
    cfg = zh.config(64, 32, [layer])
    folder = zh.make_folder(tmp_path, cfg, seed=9, gain=1.0, edit=_one_direction(cfg, 63))
    oracle = zh.Oracle(folder)
    toks = np.random.default_rng(1).integers(0, 63, size=400).tolist()
    toks[at] = 63
    other = list(toks)
    other[at] = 5
    moved = np.abs(oracle.logits(toks)[-1] - oracle.logits(other)[-1]).max()
    assert moved > 100 * tolerance(torch.float32, zh.like_config(cfg), None), moved
    for dtype in DTYPES:
        engine = build_engine(folder, dtype, max_tokens=512)
        compare(run_whole(engine, [toks]), oracle, [toks], dtype, cfg, f"far token {at} whole")
        compare(run_tail_by_one(engine, [toks], tail=300), oracle, [toks], dtype, cfg, f"far token {at} decoded")
        compare(run_chunked(engine, [toks], [at + 1, 2, 200, 64]), oracle, [toks], dtype, cfg, f"far token {at} portions")


def test_the_sequences_first_tokens_and_sizes_that_are_one(tmp_path):
    """Sequences of one to ten tokens (the convolutions' windows are not full, the states start at zero, a softmax of one key), and
    a model of one head, one channel, one state row, one tap and one expert."""
    cfg = zh.CONFIGS["P"]
    folder = zh.make_folder(tmp_path / "p", cfg, seed=5, gain=40.0)
    reqs = zh.random_requests(cfg, [1, 2, 3, 4, 5, 8, 10], seed=1)
    engine = build_engine(folder, torch.float32, max_tokens=64 * 7, max_seqs=7)
    compare(run_whole(engine, reqs), zh.Oracle(folder), reqs, torch.float32, cfg, "first tokens")
    compare(run_batches(engine, reqs, [list(range(7))], [1] * 7), zh.Oracle(folder), reqs, torch.float32, cfg, "first tokens, decoded together")
    ones = zh.config(40, 16, [zh.parallel((1, 1, 2, 1, zh.rot(2, 1.0)), (1, 2, 1, 1, 1, 1), mlp=zh.moe(1, 1, 1), scale=1.0),
                              zh.mamba2(1, 3, 1, 1, 1, 1, mlp=zh.dense(1))], softcap=1.0)
    folder = zh.make_folder(tmp_path / "ones", ones, seed=6, gain=4.0)
    reqs = zh.random_requests(ones, [70, 3], seed=2)
    engine = build_engine(folder, torch.float32, max_tokens=192)
    compare(run_whole(engine, reqs), zh.Oracle(folder), reqs, torch.float32, ones, "ones whole")
    compare(run_tail_by_one(engine, reqs, tail=60), zh.Oracle(folder), reqs, torch.float32, ones, "ones decoded")


def test_a_model_of_recurrent_layers_only(tmp_path):
    """A cache without page groups: long sequences hold nothing but their state rows, which are used again."""
    cfg = zh.config(70, 32, [zh.mamba2(2, 16, 16, 1, 4, 1, mlp=zh.dense(16)), zh.mamba2(1, 24, 8, 1, 3, 1)])
    for dtype in DTYPES:
        folder = zh.make_folder(tmp_path / str(dtype), cfg, seed=8, gain=1.0)
        oracle = zh.Oracle(folder)
        toks = zh.random_requests(cfg, [150, 20, 90], seed=9)
        engine = build_engine(folder, dtype, max_tokens=64, max_seqs=1)
        assert not engine.cache.group_keys
        for run in (run_whole(engine, toks), run_tail_by_one(engine, toks, tail=100), run_chunked(engine, toks, [63, 2, 65])):
            compare(run, oracle, toks, dtype, cfg, "recurrent only")


@pytest.mark.parametrize("window, keep_first", [(8, 0), (70, 3)])
def test_values_that_are_keys_behind_a_window(window, keep_first):
    """The attention's other options beside convolved keys as values: a ring of pages behind pinned ones, portions and single tokens,
    against the plain mechanisms put together."""
    from llaisys_b200.cache.kv import CacheConfig, PagedCache
    from llaisys_b200.config.spec import PartSpec
    from llaisys_b200.engine.context import StepContext
    from llaisys_b200.parts import build_part
    H, G, d, D, n = 4, 2, 16, 32, 260
    rng = np.random.default_rng(window)
    w = {"q": rng.normal(size=(H * d, D)) * 0.5, "k": rng.normal(size=(G * d, D)) * 0.5, "q.conv": rng.uniform(-1, 1, size=(H * d, 4)),
         "k.conv": rng.uniform(-1, 1, size=(G * d, 4)), "o": rng.normal(size=(D, H * d)) * 0.2}
    part = build_part("mixer", PartSpec("windowed_sink_attention", {
        "hidden_size": D, "num_heads": H, "num_kv_heads": G, "key_dim": d, "value_dim": d, "scale": 0.4, "window": window, "keep_first": keep_first,
        "cache_window": window, "values": "keys", "conv": 4, "value_scale": 0.5, "out_f32": True,
        "position": PartSpec("rope_leading", {"head_dim": d, "dims": 8, "base": 100.0})}), _env(torch.float32))
    part.load({k: _f32(v) for k, v in w.items()})
    part.prepare(512)
    h = rng.normal(size=(n, D))
    q, k = plain.short_conv(h @ w["q"].T, w["q.conv"]), plain.short_conv(h @ w["k"].T, w["k.conv"])
    r = {"dims": 8, "base": 100.0}
    v = k.reshape(n, G, d) * 0.5
    q, k = plain.rotate(q.reshape(n, H, d), np.arange(n), r), plain.rotate(k.reshape(n, G, d), np.arange(n), r)
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    visible = (j <= i) & ((i - j < window) | (j < keep_first))
    heads = [plain.softmax(np.where(visible, q[:, a] @ k[:, a // 2].T * 0.4, -np.inf)) @ v[:, a // 2] for a in range(H)]
    want = np.concatenate(heads, axis=1) @ w["o"].T
    users = part.cache_users()
    cache = PagedCache([u[0] for u in users], [None] * len(users), [u[1] for u in users], CacheConfig(max_tokens=512, max_seqs=2), torch.float32, DEV)
    for cuts in ([n], [63, 2, 65, 1, 64, 1000], [1]):
        slot, at, c = cache.acquire(), 0, 0
        while at < n:
            m = min(cuts[min(c, len(cuts) - 1)], n - at)
            c += 1
            cache.book.reserve(slot, m)
            shape = StepContext.shape_of(cache, [slot], [m], [], False)
            ctx = StepContext(cache, DEV, *shape, torch.zeros(1, dtype=torch.int32, device=DEV))
            ctx.load([slot], [m], [0] * m, [])
            _close(part.forward(_f32(h[at:at + m]), ctx, 0), want[at:at + m], 2e-5, (cuts, at))
            cache.book.commit(slot, m)
            at += m
        cache.release(slot)


# ----------------------------------------------------------------------------- whole models under every schedule
class Model:
    def __init__(self, name, tmp):
        self.name, self.tmp, self._made = name, tmp, {}

    def at(self, dtype):
        if dtype not in self._made:
            cfg = zh.for_dtype(zh.CONFIGS[self.name], dtype)
            folder = zh.make_folder(self.tmp / str(dtype), cfg, seed=11, gain=zh.GAIN[dtype])
            self._made[dtype] = (cfg, folder, zh.Oracle(folder), zh.random_requests(cfg, [130, 1, 64, 65, 9, 201], seed=3))
        return self._made[dtype]


@pytest.fixture(scope="module", params=["P", "Q", "R"])
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp(f"zu{request.param}"))


def _rooms(requests):
    return sum(-(-len(r) // 64) * 64 for r in requests)


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_and_token_by_token(model, dtype):
    cfg, folder, oracle, requests = model.at(dtype)
    engine = build_engine(folder, dtype, max_tokens=max(_rooms([r]) for r in requests))
    compare(run_whole(engine, requests), oracle, requests, dtype, cfg, f"{model.name} whole")
    compare(run_tail_by_one(engine, requests, tail=10_000), oracle, requests, dtype, cfg, f"{model.name} token by token")
    compare(run_tail_by_one(engine, requests, tail=32), oracle, requests, dtype, cfg, f"{model.name} tail")
    assert not engine.cache.live_slots


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_with_pages_slots_and_state_rows_used_again(model, dtype):
    cfg, folder, oracle, requests = model.at(dtype)
    n = len(requests)
    batches = [list(range(0, n, 2)), list(range(1, n, 2))]
    prompt_lens = [max(1, len(r) - (3 + 5 * i)) for i, r in enumerate(requests)]
    room = max(_rooms([requests[r] for r in b]) for b in batches)
    engine = build_engine(folder, dtype, max_tokens=room, max_seqs=len(batches[0]))
    compare(run_batches(engine, requests, batches, prompt_lens), oracle, requests, dtype, cfg, f"{model.name} batches")
    assert not engine.cache.live_slots
    assert [p.available for p in engine.cache.book.pools] == engine.cache.group_pages
    compare(run_batches(engine, requests, batches[::-1], prompt_lens), oracle, requests, dtype, cfg, f"{model.name} batches again")


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_mixed_steps(model, dtype):
    cfg, folder, oracle, _ = model.at(dtype)
    requests = zh.random_requests(cfg, [200, 300, 129, 9], seed=41)
    engine = build_engine(folder, dtype, max_tokens=320)
    for cuts in ([1000], [70, 60, 1000], [63, 1, 64, 65, 2, 1000], [2, 280, 1000], [64], [2]):
        reqs = requests if cuts != [2] else requests[2:]
        compare(run_chunked(engine, reqs, cuts), oracle, reqs, dtype, cfg, f"{model.name} portions {cuts}")
    requests = zh.random_requests(cfg, [120, 100, 210, 33], seed=43)
    plans = [[50, 1, 1, 1, 40, 1, 0, 1], [0, 0, 90], [70, 60, 0, 40, 1, 1, 30], [1, 1, 1]]
    engine = build_engine(folder, dtype, max_tokens=_rooms(requests), max_seqs=4)
    for turn in range(2):
        compare(run_mixed(engine, requests, plans), oracle, requests, dtype, cfg, f"{model.name} mixed steps, turn {turn}")
        assert not engine.cache.live_slots
        requests, plans = requests[::-1], plans[::-1]


def test_bfloat16_does_not_depend_on_how_the_steps_are_cut(model):
    """bfloat16 logits of whole prompts (recurrence in chunks on the tensor cores), of portions, of unequal batches and of
    single tokens (recurrence token by token) agree with one another: a stale state row or a page of another sequence moves
    every later row."""
    cfg, folder, _, _ = model.at(torch.bfloat16)
    requests = zh.random_requests(cfg, [150, 70, 9], seed=2)
    engine = build_engine(folder, torch.bfloat16, max_tokens=_rooms(requests), max_seqs=3)
    whole = run_whole(engine, requests)
    for what, other in (("portions", run_chunked(engine, requests, [63, 2, 65])), ("together", run_batches(engine, requests, [[0, 1, 2]], [100, 64, 1])),
                        ("decoded", run_tail_by_one(engine, requests, tail=40))):
        off = 0
        for key, ref in whole.items():
            rms = np.sqrt((ref.astype(np.float64) ** 2).mean())
            off += np.sqrt(((other[key] - ref).astype(np.float64) ** 2).mean()) > 0.05 * rms + 1e-3
        assert off <= max(2, len(whole) // 25), (what, off, len(whole))


def test_long_decoding_through_captured_steps(tmp_path):
    """Hundreds of single-token steps from a short prompt: pages fill and new ones are taken, the states and the convolutions'
    inputs are carried through every step, and the steps are replayed from a captured graph."""
    for dtype in DTYPES:
        cfg = zh.for_dtype(zh.CONFIGS["P"], dtype)
        folder = zh.make_folder(tmp_path / str(dtype), cfg, seed=21, gain=zh.GAIN[dtype])
        oracle = zh.Oracle(folder)
        requests = zh.random_requests(cfg, [330, 290], seed=6)
        engine = build_engine(folder, dtype, max_tokens=_rooms(requests), max_seqs=2)
        assert engine.use_graphs
        compare(run_batches(engine, requests, [[0, 1]], [4, 1]), oracle, requests, dtype, cfg, "long decoding")
        assert engine.graph_replays > 250


# ----------------------------------------------------------------------------- entry points
def _greedy(oracle, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(oracle.logits(seq)[-1])))
    return seq[len(prompt):]


def test_greedy_generation_through_the_entry_point_and_scheduler(tmp_path):
    from llaisys_b200.models import CausalLM, DeviceType
    cfg = zh.CONFIGS["P"]
    folder = zh.make_folder(tmp_path, cfg, seed=31, gain=40.0)
    oracle = zh.Oracle(folder)
    model = CausalLM(folder, DeviceType.NVIDIA, dtype="float32", max_tokens=64 * 4)
    prompts = zh.random_requests(cfg, [5, 9, 2, 70, 1, 17], seed=3)
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
    folder = zh.make_folder(tmp_path / "m", zh.CONFIGS["P"], seed=17, gain=40.0)
    oracle = zh.Oracle(folder)
    (tmp_path / "batch.txt").write_text("5,17,3,200,7,7,7,7,7\n[9, 8]\n1\n")
    out = subprocess.run([sys.executable, "-m", "llaisys_b200.cli", "--model", str(folder), "--batch-file", str(tmp_path / "batch.txt"),
                          "--max_steps", "6", "--dtype", "float32", "--test"], env=env, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert out.stdout.count("Tokens:") == 3 and "Test passed" in out.stdout
    want = [5, 17, 3, 200, 7, 7, 7, 7, 7] + _greedy(oracle, [5, 17, 3, 200, 7, 7, 7, 7, 7], 6)
    assert str(want) in out.stdout or ", ".join(map(str, want)) in out.stdout, out.stdout[-1500:]
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(zh.CONFIGS["Q"]))
    out = subprocess.run([sys.executable, "-m", "llaisys_b200.cli", "--random-weights", str(cfg), "--seed", "3", "--tokens", "1,2,3",
                          "--max_steps", "4", "--dtype", "float32", "--test"], env=env, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert "Tokens:" in out.stdout and "Test passed" in out.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_of_a_trace(tmp_path, dtype):
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    cfg = zh.for_dtype(zh.CONFIGS["P"], td)
    folder = zh.make_folder(tmp_path / "m", cfg, seed=13, gain=zh.GAIN[td])
    requests = zh.random_requests(cfg, [1, 7, 90, 20], seed=8)
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
    oracle = zh.Oracle(folder)
    for step, keys in rows:
        data = np.frombuffer((out_dir / f"{step}.f32").read_bytes(), dtype="<f4").reshape(len(keys), cfg["vocab"])
        for i, (r, p) in enumerate(keys):
            ref = oracle.logits(requests[r])
            assert np.abs(data[i] - ref[p]).max() <= tolerance(td, zh.like_config(cfg), ref) * (1 if dtype == "float32" else 4), (step, r, p)

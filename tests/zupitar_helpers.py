"""Shared by the Zupitar tests: small configurations that differ from one another in every size and option, model folders
with seeded weights shaped so that a fault shows, and the plain oracle's logits."""
from __future__ import annotations

import copy
import json
from pathlib import Path

import numpy as np
import torch

import plain_qwen2
import plain_zupitar as plain


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=None, groups=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def rot(dims, base=10000.0, factor=None):
    r = {"dims": dims, "base": base}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    return r


def state_space(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def mamba2(*sizes, mlp=None):
    return {"type": "mamba2", "mixer": state_space(*sizes), "mlp": mlp}


def parallel(left, right, scales=(1.0, 1.0), mlp=None, scale=None):
    """left: (heads, kv_heads, dim, conv, rotation); right: the sizes of a state-space mixer."""
    heads, kv_heads, dim, conv, rotation = left
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else dim ** -0.5}
    if conv is not None:
        m["conv"] = conv
    if rotation:
        m["rot"] = rotation
    return {"type": "parallel", "mixer": {"left": m, "right": state_space(*right), "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def config(vocab, width, layers, softcap=None, eps=1e-5):
    c = {"architecture": "Zupitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if softcap is not None:
        c["logit_softcap"] = softcap
    return c


# P: both kinds of layer and both kinds of feed-forward, groups with and without identity experts, part of a head rotated with
#    stretched positions, unequal scales (one negative), several groups in either sense, a low cap.
# Q: sizes that are no multiples of 4 or 8 (the CUDA-core products, pieces of one element, odd unrotated rests); one tap, no
#    convolution at all, three and six taps; one query head per key head and three; no rotation, no cap, no scaling, no
#    feed-forward; identity experts without groups.
# R: heads of 64, 128 and 48 (tcgen05 and mma.sync attention), whole heads rotated; state-space heads of 64 and 72 value channels
#    and 128, 136 and 16 state rows (a second tile of columns, odd blocks of rows).
CONFIGS = {
    "P": config(211, 64, [
        parallel((4, 2, 16, 4, rot(12, 2000.0, 4.0)), (4, 8, 16, 2, 4, 2), (1.3, -0.7), dense(40)),
        mamba2(6, 16, 24, 3, 4, 3, mlp=moe(7, 3, 24, 2, (3, 2))),
        parallel((6, 2, 24, 4, rot(8, 500.0)), (2, 24, 8, 1, 4, 4), (0.6, 1.5), moe(6, 3, 16, None, (2, 1))),
        mamba2(2, 32, 40, 2, 3, 1),
    ], softcap=3.0),
    "Q": config(150, 44, [
        parallel((3, 1, 7, 3, rot(4, 300.0)), (3, 5, 6, 3, 1, 1), (0.9, 1.1), dense(20)),
        parallel((2, 2, 18, None, None), (2, 9, 13, 1, 6, 2), (1.0, 1.0)),
        mamba2(3, 7, 33, 1, 3, 7, mlp=moe(3, 2, 12, 2)),
        parallel((3, 3, 10, 1, rot(10, 50.0, 2.5)), (1, 1, 1, 1, 2, 1), (2.0, 0.5), dense(14)),
    ], eps=1e-6),
    "R": config(97, 64, [
        parallel((2, 1, 64, 4, rot(64, 100000.0)), (2, 64, 128, 1, 4, 1), (1.0, 0.5), dense(64)),
        mamba2(1, 72, 136, 1, 4, 3, mlp=moe(4, 3, 64, 4, (4, 2))),
        parallel((4, 2, 128, 4, rot(64, 1000.0, 8.0)), (4, 16, 16, 4, 4, 4), (0.5, 2.0), moe(3, 1, 32)),
        parallel((3, 3, 48, 2, rot(32, 300.0)), (2, 8, 256, 2, 4, 2), (1.5, 1.0), dense(48)),
    ], softcap=10.0),
}

GAIN = {torch.float32: 40.0, torch.bfloat16: 15.0}


def variant(cfg: dict, edit) -> dict:
    c = copy.deepcopy(cfg)
    edit(c)
    return c


def for_dtype(cfg: dict, dtype) -> dict:
    """Under bfloat16 every expert is chosen: which experts a token uses must not hang on 16-bit rounding of the stream
    (sparse routing in 16 bits is covered where both sides get the same input)."""
    if dtype != torch.bfloat16:
        return cfg

    def all_experts(c):
        for l in c["layers"]:
            if l["mlp"] and l["mlp"]["kind"] == "moe":
                r = l["mlp"]["router"]
                r["top"] = r["experts"] + r.get("identity", 0)
                if r.get("groups"):
                    r["groups"]["keep"] = r["groups"]["count"]
    return variant(cfg, all_experts)


def make_folder(tmp, cfg: dict, seed: int, gain: float, store="bfloat16", edit=None) -> Path:
    """Seeded random weights, then: the attention's query and key matrices scaled by `gain` (together) so that scores spread; taps of
    both signs and biases of the convolutions; decays between almost one and almost zero, steps and skips of both sizes; input
    matrices scaled so that silu and softplus leave their linear range; router matrices scaled so that the softmax is not flat,
    corrections of both signs, many of them larger than a score; norm weights spread; embeddings and head of size one.
    `edit` (dict of tensors -> None) changes the result further."""
    from llaisys_b200.weights import SafetensorsFile, write_random_model, write_safetensors
    folder = write_random_model(Path(tmp), cfg, seed, store)
    f = SafetensorsFile(folder / "model.safetensors")
    rng = np.random.default_rng(seed + 1)
    out = {}
    for name in f.entries:
        t = f.get(name).clone()

        def uniform(lo, hi):
            return torch.from_numpy(np.asarray(rng.uniform(lo, hi, size=tuple(t.shape)))).to(t.dtype)

        def scaled(c):
            return (t.float() * c).to(t.dtype)

        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm1b", "norm2", "norm2b"):
            t = uniform(0.5, 1.5)
        elif leaf == "conv":
            t = uniform(-0.8, 0.8)
        elif name.endswith("conv.b"):
            t = uniform(-0.5, 0.5)
        elif leaf == "A_log":
            t = uniform(-4.0, 1.0)
        elif leaf == "dt_bias":
            t = uniform(-3.0, 1.0)
        elif leaf == "D":
            t = uniform(-1.0, 1.0)
        elif leaf == "in":
            t = scaled(8.0)
        elif leaf in ("q", "k"):
            t = scaled(gain ** 0.5)
        elif leaf == "correction":
            t = uniform(-0.4, 0.1)
        elif leaf == "router":
            t = scaled(8.0)
        elif ".mlp." in name:
            t = scaled(8.0)
        elif name == "embed":
            t = scaled(50.0)
        elif name == "head":
            t = scaled(7.0)
        elif leaf == "o":
            t = scaled(4.0)
        out[name] = t
    if edit:
        edit(out)
    write_safetensors(folder / "model.safetensors", out)
    return folder


class Oracle:
    """Plain logits of whole requests, computed once per request."""

    def __init__(self, folder):
        self.config = json.loads((Path(folder) / "config.json").read_text())
        self.weights = plain_qwen2.read_safetensors(Path(folder) / "model.safetensors")
        self._memo = {}

    def logits(self, tokens) -> np.ndarray:
        key = tuple(tokens)
        if key not in self._memo:
            self._memo[key] = plain.forward(self.config, self.weights, list(tokens))[0]
        return self._memo[key]


def like_config(cfg: dict) -> dict:
    """What helpers.tolerance reads.  Its bfloat16 bound counts six roundings to 16 bits a layer; a layer of this design has
    about twice as many (two mixers, each with a convolution of its own), so it counts twice."""
    return {"num_hidden_layers": 2 * len(cfg["layers"])}


def random_requests(cfg: dict, lengths, seed: int):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]


def compare(got, oracle, requests, dtype, cfg, what=""):
    """float32: every logits row within the absolute bound of helpers.tolerance.  bfloat16: no row beyond four bounds and
    at most one row in ten beyond one (a fault, a lost key or a stale state, moves whole ranges of positions by far more).
    Models with parts of fewer than 16 channels under a norm: no row beyond eight (such a norm magnifies 16-bit rounding
    where so short a vector is small by cancellation)."""
    import helpers
    like = like_config(cfg)
    if dtype == torch.float32:
        return helpers.compare(got, oracle, requests, dtype, like, what)
    ratios = []
    for r, toks in enumerate(requests):
        ref = oracle.logits(toks)
        tol = helpers.tolerance(dtype, like, ref)
        for p in range(len(toks)):
            assert (r, p) in got, f"{what}: no logits for request {r} position {p}"
            err = float(np.abs(got[(r, p)].astype(np.float64) - ref[p]).max())
            assert np.isfinite(err), f"{what}: non-finite logits at request {r} position {p}"
            ratios.append((err / tol, r, p))
    worst = max(ratios)
    mixers = [l["mixer"].get("right", l["mixer"]) for l in cfg["layers"]]
    most = 8.0 if any(m["heads"] * m["vdim"] // m["norm_groups"] < 16 for m in mixers) else 4.0
    over = sum(1 for x in ratios if x[0] > 1.0)
    assert worst[0] <= most, f"{what}: request {worst[1]} position {worst[2]} is {worst[0]:.1f} bounds off"
    assert over <= max(1, len(ratios) // 10), f"{what}: {over} of {len(ratios)} rows are beyond the bound (worst {worst[0]:.1f} at {worst[1:]})"
    return worst[0], worst[1:]

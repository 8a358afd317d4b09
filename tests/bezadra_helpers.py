"""Shared by the Bezadra tests: small configurations that differ from one another in every size and option, model folders
with seeded weights shaped so that a fault shows, and the plain oracle's logits."""
from __future__ import annotations

import copy
import json
from pathlib import Path

import numpy as np
import torch

import plain_bezadra as plain
import plain_qwen2


def dense(ff, limit=None):
    m = {"kind": "dense", "ff": ff}
    if limit is not None:
        m["limit"] = limit
    return m


def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, softcap=None, rotation=None, mlp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if softcap is not None:
        m["softcap"] = softcap
    if rotation:
        m["rot"] = rotation
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(vocab, width, layers, loop=None, embed_scale=None, logit_scale=None, eps=1e-5):
    c = {"architecture": "Bezadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if embed_scale is not None:
        c["embedding"] = {"scale": embed_scale}
    if logit_scale is not None:
        c["logit_scale"] = logit_scale
    return c


# P: both kinds of layer, a loop of two layers run three times with layers before and after it, heads that share query/key
#    heads in both kinds, values wider than keys, part of a head rotated with wavelengths on all three sides of the
#    rescaling, a low cap, a layer without a feed-forward.
# Q: sizes that are no multiples of 4 or 8 (the CUDA-core products, heads 32 apart); one tap, three taps and six; one
#    query/key head for three value heads, as many as heads elsewhere; no rotation, no cap, no limit, no loop, no scales.
# R: heads of 64 and 128 (the tensor-core attention, convolution rows of whole 16-byte pieces), of 48 (mma.sync) and
#    a recurrent head of 130 key channels; whole heads rotated without rescaling; a loop over all layers that runs once.
CONFIGS = {
    "P": config(211, 64, [
        delta(4, 2, 16, 24, 4, dense(40, 0.8)),
        attention(4, 2, 16, 24, softcap=6.0, rotation=rot(12, 2000.0, (4.0, 1.0, 4.0, 64)), mlp=dense(24, 1.5)),
        delta(2, 2, 24, 16, 4),
        attention(2, 1, 24, 8, softcap=20.0, rotation=rot(24, 500.0), mlp=dense(32)),
    ], loop=(1, 3, 3), embed_scale=3.0, logit_scale=0.5),
    "Q": config(150, 44, [
        attention(3, 3, 18, 10, mlp=dense(20)),
        delta(3, 1, 6, 9, 3, dense(14)),
        delta(2, 2, 33, 35, 1),
        delta(1, 1, 17, 7, 6, dense(30, 0.5)),
    ], eps=1e-6),
    "R": config(97, 64, [
        delta(2, 1, 64, 64, 4, dense(64, 2.0)),
        attention(2, 1, 64, 64, softcap=10.0, rotation=rot(64, 100000.0), mlp=dense(48, 1.0)),
        delta(1, 1, 130, 128, 4),
        attention(2, 2, 48, 48, softcap=30.0, rotation=rot(32, 300.0, (8.0, 2.0, 2.0, 32)), mlp=dense(64, 1.0)),
        delta(2, 2, 128, 40, 2, dense(16, 3.0)),
    ], loop=(0, 5, 1), embed_scale=0.5, logit_scale=2.0),
}

GAIN = {torch.float32: 40.0, torch.bfloat16: 20.0}


def variant(cfg: dict, edit) -> dict:
    c = copy.deepcopy(cfg)
    edit(c)
    return c


def make_folder(tmp, cfg: dict, seed: int, gain: float, store="bfloat16", edit=None) -> Path:
    """Seeded random weights, then: the attention's queries and keys scaled by `gain` (together) so that scores spread and
    meet the cap; sinks of both signs; gates, step sizes and bottlenecks scaled so that sigmoids leave their linear range;
    decays between almost one and almost zero; taps of both signs; feed-forward matrices scaled so that the limits are met;
    norm weights spread; the re-entry matrix scaled so that it keeps the stream's size, offsets of the stream's size; the
    table scaled so that logits are of size one.  `edit` (dict of tensors -> None) changes the result further."""
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
        recurrent = ".mix." in name and cfg["layers"][int(name[1:name.index(".")])]["type"] == "channel_delta"
        if leaf == "norm1" or name == "final.norm" or leaf == "norm":
            t = uniform(0.5, 1.5)
        elif leaf == "conv":
            t = uniform(-0.8, 0.8)
        elif leaf == "A_log":
            t = uniform(-3.0, 1.5)
        elif leaf == "dt_bias":
            t = uniform(-3.0, 1.0)
        elif leaf == "sink":
            t = uniform(-2.0, 3.0)
        elif leaf in ("a1", "g1", "a2", "g2"):
            t = scaled(15.0)
        elif leaf in ("b", "g"):
            t = scaled(15.0)
        elif leaf in ("q", "k", "v") and recurrent:
            t = scaled(8.0)
        elif leaf in ("q", "k"):
            t = scaled(gain ** 0.5)
        elif ".mlp." in name:
            t = scaled(6.0)
        elif name == "loop.in":
            t = scaled(5.0)
        elif name == "loop.step":
            t = scaled(20.0)
        elif name == "embed":
            t = scaled(8.0)
        elif leaf in ("v", "o"):
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
    """What helpers.tolerance reads: layer runs (looped layers count once per pass) and, for the bfloat16 bound, one more
    layer per pass for the re-entry's product."""
    return {"num_hidden_layers": len(plain.run_order(cfg)) + (cfg["loop"]["times"] if cfg.get("loop") else 0)}


def random_requests(cfg: dict, lengths, seed: int):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]


def compare(got, oracle, requests, dtype, cfg, what=""):
    """float32: every logits row within the absolute bound of helpers.tolerance.  bfloat16: no row beyond four bounds and
    at most one row in ten beyond one (a fault, a lost key or a stale state, moves whole ranges of positions by far more).
    Models with recurrent heads of fewer than 16 value channels: no row beyond eight (a head's result is normed over its
    channels, which magnifies 16-bit rounding where so short a vector is small by cancellation; the rows in question are
    bit-equal between whole prompts, single tokens and mixed steps)."""
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
    most = 8.0 if any(l["type"] == "channel_delta" and l["mixer"]["vdim"] < 16 for l in cfg["layers"]) else 4.0
    over = sum(1 for x in ratios if x[0] > 1.0)
    assert worst[0] <= most, f"{what}: request {worst[1]} position {worst[2]} is {worst[0]:.1f} bounds off"
    assert over <= max(1, len(ratios) // 10), f"{what}: {over} of {len(ratios)} rows are beyond the bound (worst {worst[0]:.1f} at {worst[1:]})"
    return worst[0], worst[1:]

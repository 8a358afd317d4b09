"""Typed configuration of the Bezadra decoder, read from its own config.json keys.

    architecture    "Bezadra"
    vocab, width    vocabulary and stream width
    embedding       {scale} (absent: 1)
    norm            {eps}
    logit_scale     what the logits are multiplied by (1 when absent)
    loop            {start, stop, times}: the layers start .. stop - 1 run `times` times in a row (absent: once)
    layers          list of {type: "channel_delta" | "attention", mixer: {...}, mlp: {...} or null}
      channel_delta mixer   heads, kv_heads (query/key heads), dim, vdim, conv (taps of the short convolutions)
      attention mixer       heads, kv_heads, dim, vdim, scale, softcap (optional),
                            rot: {dims, base, scaling: {factor, low, high, original} (optional)} (optional)
      mlp                   {kind: "dense", ff, limit (optional)}
      (kv_heads absent: as many as heads; vdim absent: as wide as dim)

Tensor names: embed (also the output matrix), loop.in, loop.step, l<i>.norm1, l<i>.mix.*, l<i>.mlp.{gate, up, down},
final.norm.

A layer is `shared_norm_parallel`: its mixer and its feed-forward read one normed stream and both join it.  Every norm is a
layer norm with a weight and no bias.  Each pass over the looped layers is an entry of the run order with a cache and a
state of its own; the entry that opens a pass first replaces the stream by a projection of the stream and the embedding's
output side by side, plus the pass's offset.  The configuration names no longest sequence; MAX_POSITIONS is this library's
bound.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .registry import register_architecture
from .spec import CallSpec, ConfigError, LayerSpec, ModelSpec, PartSpec, SubLayerSpec
from .vumezen import _dict, _float, _int

MAX_POSITIONS = 1 << 18
SWISH_ALPHA = 1.702           # the feed-forward's activation is g * sigmoid(1.702 g): the design fixes the constant
DECAY_RANK = 16               # bottleneck of the decay and of the output gate in random weights (a file's own size is read from it)


@dataclass(frozen=True)
class BezadraRotation:
    dims: int
    base: float
    wave: Optional[Dict[str, float]]


@dataclass(frozen=True)
class BezadraDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class BezadraAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot: Optional[BezadraRotation]


@dataclass(frozen=True)
class BezadraMLP:
    ff: int
    limit: float


def _rotation(m: dict, where: str, dim: int) -> Optional[BezadraRotation]:
    if m.get("rot") is None:
        return None
    rot = _dict(m, "rot", where)
    dims = _int(rot, "dims", f"{where}.rot", 0)
    if dims == 0:
        return None
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}: rot.dims={dims} must be even and at most dim={dim}")
    wave = None
    if rot.get("scaling") is not None:
        s, w = _dict(rot, "scaling", f"{where}.rot"), f"{where}.rot.scaling"
        wave = {k: _float(s, k, w) for k in ("factor", "low", "high", "original")}
        if wave["high"] < wave["low"]:
            raise ConfigError(f"{w}: high={wave['high']} must not lie below low={wave['low']}")
    return BezadraRotation(dims=dims, base=_float(rot, "base", f"{where}.rot"), wave=wave)


def _mixer(kind, m: dict, where: str):
    if kind not in ("channel_delta", "attention"):
        raise ConfigError(f"{where}: the mixers of this architecture are 'channel_delta' and 'attention', got {kind!r}")
    heads = _int(m, "heads", where)
    kv_heads = _int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads cannot share {kv_heads} key heads")
    dim = _int(m, "dim", where)
    vdim = _int(m, "vdim", where) if m.get("vdim") is not None else dim
    if kind == "channel_delta":
        return BezadraDelta(heads, kv_heads, dim, vdim, taps=_int(m, "conv", where))
    return BezadraAttention(heads, kv_heads, dim, vdim, scale=_float(m, "scale", where, positive=False),
                            softcap=_float(m, "softcap", where) if m.get("softcap") is not None else None,
                            rot=_rotation(m, where, dim))


def _mlp(mlp, where: str) -> Optional[BezadraMLP]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    if mlp.get("kind") != "dense":
        raise ConfigError(f"{where}: the feed-forward of this architecture is kind 'dense', got {mlp.get('kind')!r}")
    limit = _float(mlp, "limit", where) if mlp.get("limit") is not None else float("inf")       # no limit: nothing is clamped
    return BezadraMLP(ff=_int(mlp, "ff", where), limit=limit)


@register_architecture("Bezadra")
@dataclass(frozen=True)
class BezadraConfig:
    vocab: int
    width: int
    embed_scale: float
    eps: float
    logit_scale: float
    loop: Optional[Tuple[int, int, int]]      # (start, stop, times)
    mixers: Tuple[Any, ...]                   # BezadraDelta or BezadraAttention per layer
    ffs: Tuple[Any, ...]                      # BezadraMLP or None per layer
    raw: Any = None

    @classmethod
    def from_dict(cls, d: dict) -> "BezadraConfig":
        vocab, width = _int(d, "vocab", "config"), _int(d, "width", "config")
        eps = _float(_dict(d, "norm", "config"), "eps", "norm")
        scale = 1.0
        if d.get("embedding") is not None and _dict(d, "embedding", "config").get("scale") is not None:
            scale = _float(d["embedding"], "scale", "embedding", positive=False)
        logit_scale = _float(d, "logit_scale", "config", positive=False) if d.get("logit_scale") is not None else 1.0
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config: 'layers' must be a non-empty list")
        mixers, ffs = [], []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict):
                raise ConfigError(f"{where} must be an object")
            mixers.append(_mixer(layer.get("type"), _dict(layer, "mixer", where), where))
            ffs.append(_mlp(layer.get("mlp"), f"{where}.mlp"))
        loop = None
        if d.get("loop") is not None:
            lp = _dict(d, "loop", "config")
            loop = (_int(lp, "start", "loop", 0), _int(lp, "stop", "loop"), _int(lp, "times", "loop"))
            if not (loop[0] < loop[1] <= len(layers)):
                raise ConfigError(f"loop: layers {loop[0]} .. {loop[1] - 1} do not lie among the {len(layers)} layers")
        return cls(vocab=vocab, width=width, embed_scale=scale, eps=eps, logit_scale=logit_scale, loop=loop, mixers=tuple(mixers),
                   ffs=tuple(ffs), raw=copy.deepcopy(d))

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(self.raw)

    def order(self):
        """[(layer, the pass it opens or None)] in the order the layers run."""
        n = len(self.mixers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        out = [(i, None) for i in range(start)]
        for t in range(times):
            out += [(i, t if i == start else None) for i in range(start, stop)]
        return out + [(i, None) for i in range(stop, n)]

    def to_spec(self) -> ModelSpec:
        D = self.width
        norm = {"size": D, "eps": self.eps, "tensor": ""}
        layers = []
        for i, (m, ff) in enumerate(zip(self.mixers, self.ffs)):
            p = f"l{i}"
            if isinstance(m, BezadraDelta):
                mixer = PartSpec("channel_delta_rule", {
                    "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
                    "taps": m.taps, "query_scale": m.dim ** -0.5, "eps": self.eps, "decay_rank": DECAY_RANK, "gate_rank": DECAY_RANK},
                    prefix=f"{p}.mix")
            else:
                position = None
                if m.rot is not None:
                    position = PartSpec("rope_leading", {"head_dim": m.dim, "dims": m.rot.dims, "base": m.rot.base, "wave": m.rot.wave})
                mixer = PartSpec("windowed_sink_attention", {
                    "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
                    "scale": m.scale, "window": None, "sink": "learned", "softcap": m.softcap, "gate": "elements",
                    "position": position}, prefix=f"{p}.mix")
            # the layer's one norm stands before its first sub-layer; the arrangement hands its output to both
            subs = [SubLayerSpec("mixer", mixer, PartSpec("layer_norm", norm, prefix=f"{p}.norm1"))]
            if ff is not None:
                subs.append(SubLayerSpec("ffn", PartSpec("gated_mlp", {
                    "hidden_size": D, "intermediate_size": ff.ff, "act": "swish_clamped", "limit": ff.limit, "alpha": SWISH_ALPHA,
                    "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix=f"{p}.mlp")))
            layers.append(LayerSpec("shared_norm_parallel", tuple(subs)))
        reentry = None
        if self.loop is not None:
            reentry = PartSpec("embedding_projection", {"hidden_size": D, "passes": self.loop[2], "matrix": "in", "tensor": "step"}, prefix="loop")
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D, max_positions=MAX_POSITIONS,
            embedding=PartSpec("scaled_pair_embedding", {"vocab_size": self.vocab, "hidden_size": D, "scale": self.embed_scale,
                                                         "tensor": "embed", "pair": None}),
            layers=tuple(layers),
            order=tuple(CallSpec(layer=i, opens_pass=t) for i, t in self.order()),
            final_norm=PartSpec("layer_norm", norm, prefix="final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": D, "tied_to": "embed", "scale": self.logit_scale},
                          prefix="head"),
            stop_token_ids=(), reentry=reentry)

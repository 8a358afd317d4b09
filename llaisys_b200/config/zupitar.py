"""Typed configuration of the Zupitar decoder, read from its own config.json keys.

    architecture    "Zupitar"
    vocab, width    vocabulary and stream width
    norm            {eps}
    logit_softcap   cap on the logits (absent: none)
    layers          list of {type: "parallel" | "mamba2", mixer: {...}, mlp: {...} or null}
      parallel mixer   left: heads, kv_heads, dim, vdim (as wide as dim), scale, conv (taps of the short convolutions),
                             rot: {dims, base, scaling: {factor} (optional)} (optional)
                       right: a mamba2 mixer
                       left_scale, right_scale (1 when absent)
      mamba2 mixer     heads, vdim, state, groups, conv, norm_groups
      mlp              {kind: "dense", ff} or
                       {kind: "moe", router: {experts, top, identity (optional), groups: {count, keep} (optional)}, expert: {ff}}
      (kv_heads absent: as many as heads; groups and norm_groups absent: 1)

Tensor names: embed, l<i>.norm1, l<i>.norm1b, l<i>.norm2, l<i>.norm2b, l<i>.mix.*, l<i>.mlp.*, final.norm, head.

A layer is `sandwich_residual`: each part sits between an RMS norm of its input and one of its output.  A parallel mixer adds an
attention whose values are its convolved keys and a state-space mixer, each times a constant.  The router's softmax, groups and
choice run over the experts and, behind them, the identity experts.  The configuration names no longest sequence; MAX_POSITIONS
is this library's bound.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .registry import register_architecture
from .spec import CallSpec, ConfigError, LayerSpec, ModelSpec, PartSpec, SubLayerSpec
from .vumezen import _dict, _float, _int

MAX_POSITIONS = 1 << 18


@dataclass(frozen=True)
class ZupitarAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    taps: Optional[int]
    rot: Optional[Tuple[int, float, float]]       # dims, base, factor


@dataclass(frozen=True)
class ZupitarMamba:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class ZupitarParallel:
    left: ZupitarAttention
    right: ZupitarMamba
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class ZupitarDense:
    ff: int


@dataclass(frozen=True)
class ZupitarMoE:
    experts: int
    top: int
    identity: int
    groups: Optional[Tuple[int, int]]
    ff: int


def _rotation(m: dict, where: str, dim: int) -> Optional[Tuple[int, float, float]]:
    if m.get("rot") is None:
        return None
    rot = _dict(m, "rot", where)
    dims = _int(rot, "dims", f"{where}.rot", 0)
    if dims == 0:
        return None
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}: rot.dims={dims} must be even and at most dim={dim}")
    factor = 1.0
    if rot.get("scaling") is not None:
        factor = _float(_dict(rot, "scaling", f"{where}.rot"), "factor", f"{where}.rot.scaling")
    return dims, _float(rot, "base", f"{where}.rot"), factor


def _attention(m: dict, where: str) -> ZupitarAttention:
    heads = _int(m, "heads", where)
    kv_heads = _int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} query heads cannot share {kv_heads} key/value heads")
    dim = _int(m, "dim", where)
    if m.get("vdim") is not None and _int(m, "vdim", where) != dim:
        raise ConfigError(f"{where}: the values are the keys, so vdim={m['vdim']} must be dim={dim}")
    return ZupitarAttention(heads, kv_heads, dim, _float(m, "scale", where, positive=False),
                            taps=_int(m, "conv", where) if m.get("conv") is not None else None, rot=_rotation(m, where, dim))


def _mamba(m: dict, where: str) -> ZupitarMamba:
    heads, vdim, state = _int(m, "heads", where), _int(m, "vdim", where), _int(m, "state", where)
    groups = _int(m, "groups", where) if m.get("groups") is not None else 1
    norm_groups = _int(m, "norm_groups", where) if m.get("norm_groups") is not None else 1
    if heads % groups:
        raise ConfigError(f"{where}: {heads} heads cannot share {groups} groups")
    if (heads * vdim) % norm_groups:
        raise ConfigError(f"{where}: {heads * vdim} channels cannot be normed in norm_groups={norm_groups} equal parts")
    return ZupitarMamba(heads, vdim, state, groups, _int(m, "conv", where), norm_groups)


def _mixer(kind, m: dict, where: str):
    if kind == "mamba2":
        return _mamba(m, where)
    if kind == "parallel":
        scale = lambda k: _float(m, k, where, positive=False) if m.get(k) is not None else 1.0
        return ZupitarParallel(_attention(_dict(m, "left", where), f"{where}.left"), _mamba(_dict(m, "right", where), f"{where}.right"),
                               scale("left_scale"), scale("right_scale"))
    raise ConfigError(f"{where}: the mixers of this architecture are 'parallel' and 'mamba2', got {kind!r}")


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    if mlp.get("kind") == "dense":
        return ZupitarDense(ff=_int(mlp, "ff", where))
    if mlp.get("kind") != "moe":
        raise ConfigError(f"{where}: the feed-forward of this architecture is kind 'dense' or 'moe', got {mlp.get('kind')!r}")
    router = _dict(mlp, "router", where)
    experts, top = _int(router, "experts", f"{where}.router"), _int(router, "top", f"{where}.router")
    identity = _int(router, "identity", f"{where}.router", 0) if router.get("identity") is not None else 0
    if top > experts + identity:
        raise ConfigError(f"{where}: a token cannot use {top} of {experts + identity} experts")
    groups = None
    if router.get("groups") is not None:
        g, w = _dict(router, "groups", f"{where}.router"), f"{where}.router.groups"
        count, keep = _int(g, "count", w), _int(g, "keep", w)
        if (experts + identity) % count or keep > count or keep * ((experts + identity) // count) < top:
            raise ConfigError(f"{where}: {experts + identity} experts in {count} groups of which {keep} are kept cannot give {top} choices")
        groups = (count, keep)
    return ZupitarMoE(experts, top, identity, groups, ff=_int(_dict(mlp, "expert", where), "ff", f"{where}.expert"))


@register_architecture("Zupitar")
@dataclass(frozen=True)
class ZupitarConfig:
    vocab: int
    width: int
    eps: float
    softcap: Optional[float]
    mixers: Tuple[Any, ...]                   # ZupitarParallel or ZupitarMamba per layer
    ffs: Tuple[Any, ...]                      # ZupitarDense, ZupitarMoE or None per layer
    raw: Any = None

    @classmethod
    def from_dict(cls, d: dict) -> "ZupitarConfig":
        vocab, width = _int(d, "vocab", "config"), _int(d, "width", "config")
        eps = _float(_dict(d, "norm", "config"), "eps", "norm")
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
        return cls(vocab=vocab, width=width, eps=eps, softcap=_float(d, "logit_softcap", "config") if d.get("logit_softcap") is not None else None,
                   mixers=tuple(mixers), ffs=tuple(ffs), raw=copy.deepcopy(d))

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(self.raw)

    def _mamba_spec(self, m: ZupitarMamba, prefix: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("state_space", {
            "hidden_size": self.width, "num_heads": m.heads, "value_dim": m.vdim, "state": m.state, "groups": m.groups, "taps": m.taps,
            "norm_groups": m.norm_groups, "eps": self.eps, "out_scale": scale}, prefix=prefix)

    def _mixer_spec(self, m, prefix: str) -> PartSpec:
        if isinstance(m, ZupitarMamba):
            return self._mamba_spec(m, prefix)
        l = m.left
        position = None
        if l.rot is not None:
            position = PartSpec("rope_leading", {"head_dim": l.dim, "dims": l.rot[0], "base": l.rot[1], "factor": l.rot[2]})
        left = PartSpec("windowed_sink_attention", {
            "hidden_size": self.width, "num_heads": l.heads, "num_kv_heads": l.kv_heads, "key_dim": l.dim, "value_dim": l.dim,
            "scale": l.scale, "window": None, "values": "keys", "conv": l.taps, "value_scale": m.left_scale, "out_f32": True,
            "position": position}, prefix=f"{prefix}.left")
        return PartSpec("parallel_mixers", {"hidden_size": self.width, "combine": "sum", "branches": [
            {"part": left}, {"part": self._mamba_spec(m.right, f"{prefix}.right", m.right_scale)}]}, prefix=prefix)

    def _ffn_spec(self, ff, prefix: str) -> PartSpec:
        if isinstance(ff, ZupitarDense):
            return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": ff.ff, "act": "relu",
                                          "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix=prefix)
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": ff.experts, "top": ff.top, "identity": ff.identity, "expert_ff": ff.ff,
            "gate": "softmax", "act": "silu", "groups": {"count": ff.groups[0], "keep": ff.groups[1]} if ff.groups else None,
            "group_score": "max", "shared_ff": None, "use_bias": True}, prefix=prefix)

    def to_spec(self) -> ModelSpec:
        D = self.width
        norm = lambda name: PartSpec("rms_norm", {"size": D, "eps": self.eps, "tensor": ""}, prefix=name)
        layers = []
        for i, (m, ff) in enumerate(zip(self.mixers, self.ffs)):
            p = f"l{i}"
            subs = [SubLayerSpec("mixer", self._mixer_spec(m, f"{p}.mix"), norm(f"{p}.norm1"), norm(f"{p}.norm1b"))]
            if ff is not None:
                subs.append(SubLayerSpec("ffn", self._ffn_spec(ff, f"{p}.mlp"), norm(f"{p}.norm2"), norm(f"{p}.norm2b")))
            layers.append(LayerSpec("sandwich_residual", tuple(subs), {"mult": 1.0}))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D, max_positions=MAX_POSITIONS,
            embedding=PartSpec("scaled_pair_embedding", {"vocab_size": self.vocab, "hidden_size": D, "scale": 1.0, "tensor": "embed", "pair": None}),
            layers=tuple(layers), order=tuple(CallSpec(layer=i) for i in range(len(layers))),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": D, "tied_to": None, "tensor": "", "softcap": self.softcap},
                          prefix="head"),
            stop_token_ids=())

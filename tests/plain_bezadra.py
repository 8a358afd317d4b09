"""A plain, slow evaluation of the Bezadra decoder in float64 numpy: one function per mechanism, whole sequences, no
cache, no code shared with the package.  `forward(config, tensors, tokens)` takes the parsed config.json, a dict of
arrays by tensor name and one sequence's token ids; it returns the logits at every position and the residual stream
after every layer run.

Notation: T tokens, stream width D, h a layer's normed input, positions p = 0 .. T-1.
"""
from __future__ import annotations

import math

import numpy as np

UNIT_EPS = 1e-6          # inside the root of the unit vectors
ALPHA = 1.702            # of the feed-forward's activation


def layer_norm(x, w, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)


def short_conv(x, w):
    """x [T, C], w [C, taps]: out[t, c] = sum_j w[c, j] x[t - (taps - 1) + j, c], zeros before the first token."""
    T, taps = x.shape[0], w.shape[1]
    out = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += x[:T - back] * w[:, j]
    return out


def channel_decay(h, w, heads, dim):
    """g [T, heads, dim]: exp(-exp(A) softplus(Wa2 (Wa1 h) + b)), one A per head."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    return np.exp(-np.exp(w["A_log"])[:, None] * softplus(z).reshape(len(h), heads, dim))


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, d]; v [T, H, dv]; beta [T, H].  Per head S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T;
    o = S^T q."""
    T, H, d = k.shape
    S = np.zeros((H, d, v.shape[-1]))
    o = np.zeros(v.shape)
    for t in range(T):
        S = S * g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    return o


def delta_inputs(h, w, m):
    """What enters the recurrence, query and key heads already given to the value heads they serve."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(h @ w["q"].T, w["q.conv"])).reshape(T, G, d)
    k = silu(short_conv(h @ w["k"].T, w["k.conv"])).reshape(T, G, d)
    v = silu(short_conv(h @ w["v"].T, w["v.conv"])).reshape(T, H, dv)
    own = np.arange(H) // (H // G)
    return (unit(q) * d ** -0.5)[:, own], unit(k)[:, own], v, channel_decay(h, w, H, d), sigmoid(h @ w["b"].T)


def channel_delta(h, w, m, eps):
    T, H, dv = h.shape[0], m["heads"], m["vdim"]
    o = delta_rule(*delta_inputs(h, w, m))
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, dv)
    return (rms(o, eps) * w["norm"] * gate).reshape(T, H * dv) @ w["o"].T


def frequencies(rot):
    """base^(-2i/dims), rescaled by wavelength where the rotation asks for it: short waves keep their frequency, long ones
    are divided by the factor, a linear blend between."""
    f = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for x in f:
        wave = 2.0 * math.pi / x
        if wave < s["original"] / s["high"]:
            out.append(x)
        elif wave > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            c = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - c) * x / s["factor"] + c * x)
    return np.array(out)


def rotate(x, pos, rot):
    """x [T, n, d]: element i of the first `dims` turned with element i + dims/2."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    ang = np.asarray(pos, dtype=np.float64)[:, None] * frequencies(rot)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def sink_softmax(s, sink):
    """Causal softmax over the rows of s [T, T] whose denominator has the extra term exp(sink)."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def capped(s, cap):
    return s if not cap else cap * np.tanh(s / cap)


def attention(h, w, m, pos=None):
    T = h.shape[0]
    pos = np.arange(T) if pos is None else pos
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w["q"].T).reshape(T, H, d), pos, m.get("rot"))
    k = rotate((h @ w["k"].T).reshape(T, G, d), pos, m.get("rot"))
    v = (h @ w["v"].T).reshape(T, G, dv)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        kv = hd // (H // G)
        out[:, hd] = sink_softmax(capped((q[:, hd] @ k[:, kv].T) * m["scale"], m.get("softcap")), w["sink"][hd]) @ v[:, kv]
    return (out.reshape(T, H * dv) * sigmoid(h @ w["g"].T)) @ w["o"].T


def feed_forward(h, w, mlp):
    limit = np.inf if mlp.get("limit") is None else mlp["limit"]
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(ALPHA * g) * (u + 1.0)) @ w["down"].T


def sub(tensors, prefix):
    return {k[len(prefix) + 1:]: v for k, v in tensors.items() if k.startswith(prefix + ".")}


def layer(x, i, cfg, tensors):
    eps, L = cfg["norm"]["eps"], cfg["layers"][i]
    w = sub(tensors, f"l{i}.mix")
    h = layer_norm(x, tensors[f"l{i}.norm1"], eps)
    y = channel_delta(h, w, L["mixer"], eps) if L["type"] == "channel_delta" else attention(h, w, L["mixer"])
    if L.get("mlp") is not None:
        y = y + feed_forward(h, sub(tensors, f"l{i}.mlp"), L["mlp"])
    return x + y


def run_order(cfg):
    """[(layer, pass number or None when the layer does not open a pass)] in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, tensors, tokens):
    tensors = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x0 = tensors["embed"][np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    x, after = x0, []
    for i, t in run_order(cfg):
        if t is not None:
            x = np.concatenate([x, x0], axis=-1) @ tensors["loop.in"].T + tensors["loop.step"][t]
        x = layer(x, i, cfg, tensors)
        after.append(x)
    h = layer_norm(x, tensors["final.norm"], cfg["norm"]["eps"])
    return (h @ tensors["embed"].T) * cfg.get("logit_scale", 1.0), np.stack(after)

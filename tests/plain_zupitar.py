"""A plain, slow evaluation of the Zupitar decoder in float64 numpy: one function per mechanism, whole sequences, no
cache, no code shared with the package.  `forward(config, tensors, tokens)` takes the parsed config.json, a dict of
arrays by tensor name and one sequence's token ids; it returns the logits at every position and the residual stream
after every layer.

Notation: T tokens, stream width D, h a part's normed input, positions p = 0 .. T-1.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def short_conv(x, w, bias=None):
    """x [T, C], w [C, taps]: out[t, c] = bias[c] + sum_j w[c, j] x[t - (taps - 1) + j, c], zeros before the first token."""
    T, taps = x.shape[0], w.shape[1]
    out = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += x[:T - back] * w[:, j]
    return out if bias is None else out + bias


def rotate(x, pos, rot):
    """x [T, n, d]: element i of the first `dims` turned with element i + dims/2 by pos * base^(-2i/dims) / factor."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    freq = rot["base"] ** (-2.0 * np.arange(half) / rot["dims"]) / (rot.get("scaling") or {"factor": 1.0})["factor"]
    ang = np.asarray(pos, dtype=np.float64)[:, None] * freq[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def causal_softmax(s):
    T = s.shape[0]
    return softmax(np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf))


def attention(h, w, m, pos=None):
    """Convolved queries and keys; the values are the convolved keys as they are before the rotation."""
    T = h.shape[0]
    pos = np.arange(T) if pos is None else pos
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w["q"].T, h @ w["k"].T
    if m.get("conv"):
        q, k = short_conv(q, w["q.conv"]), short_conv(k, w["k.conv"])
    v = k.reshape(T, G, d)
    q, k = rotate(q.reshape(T, H, d), pos, m.get("rot")), rotate(v, pos, m.get("rot"))
    out = np.zeros((T, H, d))
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = causal_softmax((q[:, hd] @ k[:, g].T) * m["scale"]) @ v[:, g]
    return out.reshape(T, H * d) @ w["o"].T


def state_space(x, B, C, dt, A, D):
    """x [T, H, P]; B, C [T, H, N]; dt [T, H]; A, D [H].  Per head S <- exp(A dt) S + dt B x^T, y = S^T C + D x."""
    T, H, P = x.shape
    S = np.zeros((H, B.shape[-1], P))
    y = np.zeros((T, H, P))
    for t in range(T):
        S = np.exp(A * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t]
    return y


def state_space_inputs(h, w, m):
    """(z [T, inner], x, B, C and dt as they enter the recurrence, B and C already given to the heads of their group)."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ w["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w["conv"], w["conv.b"]))
    own = np.arange(H) // (H // G)
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)[:, own]
    C = xbc[:, inner + G * N:].reshape(T, G, N)[:, own]
    return z, x, B, C, softplus(dt + w["dt_bias"])


def gated_group_norm(y, z, weight, groups, eps):
    """y * silu(z), each of `groups` equal parts of the row divided by its own root mean square, times the weight."""
    g = (y * silu(z)).reshape(len(y), groups, -1)
    return rms(g, eps).reshape(len(y), -1) * weight


def mamba2(h, w, m, eps):
    z, x, B, C, dt = state_space_inputs(h, w, m)
    y = state_space(x, B, C, dt, -np.exp(w["A_log"]), w["D"])
    return gated_group_norm(y.reshape(len(h), -1), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


def parallel(h, w, m, eps):
    return m.get("left_scale", 1.0) * attention(h, sub(w, "left"), m["left"]) + m.get("right_scale", 1.0) * mamba2(h, sub(w, "right"), m["right"], eps)


def dense(h, w):
    return (np.maximum(h @ w["gate"].T, 0.0) * (h @ w["up"].T)) @ w["down"].T


def route(z, correction, r):
    """(chosen [T, top], weights [T, top]) from the router's logits [T, experts + identity]."""
    s = softmax(z)
    choice = s + correction
    if r.get("groups"):
        count, keep = r["groups"]["count"], r["groups"]["keep"]
        c = choice.reshape(len(z), count, -1)
        best = np.argsort(-c.max(axis=-1), axis=-1, kind="stable")[:, :keep]
        kept = np.zeros((len(z), count), dtype=bool)
        np.put_along_axis(kept, best, True, axis=1)
        choice = np.where(kept[:, :, None], c, -np.inf).reshape(len(z), -1)
    idx = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    return idx, np.take_along_axis(s, idx, axis=1)


def moe(h, w, mlp):
    r = mlp["router"]
    idx, wgt = route(h @ w["router"].T, w["correction"], r)
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(idx[t], wgt[t]):
            if e >= r["experts"]:
                out[t] += a * h[t]                           # an identity expert
            else:
                out[t] += a * (w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])))
    return out


def sub(tensors, prefix):
    return {k[len(prefix) + 1:]: v for k, v in tensors.items() if k.startswith(prefix + ".")}


def layer(x, i, cfg, tensors):
    eps, L = cfg["norm"]["eps"], cfg["layers"][i]
    norm = lambda v, name: rms(v, eps) * tensors[f"l{i}.{name}"]
    mixer = {"parallel": parallel, "mamba2": mamba2}[L["type"]]
    x = x + norm(mixer(norm(x, "norm1"), sub(tensors, f"l{i}.mix"), L["mixer"], eps), "norm1b")
    if L.get("mlp") is not None:
        h, w = norm(x, "norm2"), sub(tensors, f"l{i}.mlp")
        x = x + norm(dense(h, w) if L["mlp"]["kind"] == "dense" else moe(h, w, L["mlp"]), "norm2b")
    return x


def capped(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def forward(cfg, tensors, tokens):
    tensors = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    x, after = tensors["embed"][np.asarray(tokens)], []
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, tensors)
        after.append(x)
    h = rms(x, cfg["norm"]["eps"]) * tensors["final.norm"]
    return capped(h @ tensors["head"].T, cfg.get("logit_softcap")), np.stack(after)

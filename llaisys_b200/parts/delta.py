from __future__ import annotations

import torch

from .. import kernels
from .base import Mixer, TensorDecl, register_part
from .normed_attention import _fuse


@register_part("mixer", "channel_delta_rule")
class ChannelDeltaRule(Mixer):
    """A recurrent mixer with a matrix of memory per head, S [key_dim, value_dim] in float32, that forgets per key channel and
    corrects what it holds for a key towards the token's value:

        q, k = Wq h, Wk h (num_kv_heads x key_dim), v = Wv h (num_heads x value_dim), each through a causal convolution of
        `taps` tokens per channel and silu; q and k made unit vectors per head, q times query_scale; head i works with
        query/key head i / (num_heads / num_kv_heads)
        g = exp(-exp(A_h) softplus(Wa2 (Wa1 h) + b)) per head and key channel, beta = sigmoid(Wb h) per head
        S <- diag(g) S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
        out = Wo (rms_norm(o over value_dim; weight shared by heads) * sigmoid(Wg2 (Wg1 h)))

    The sequence's memory is two users of the cache's fixed-size state (zero when the sequence starts): the matrices S, and
    the convolutions' last taps - 1 inputs.  q, k, v and beta's logits are one matrix product whose output stays float32 in
    both precisions; the two bottlenecks are a second one; everything from the convolution to o is float32.  Single tokens,
    short steps and the 32-bit path run token by token; longer steps in chunks (kernels.delta_scan).  The bottlenecks' sizes
    are the shapes of `a1` and `g1`.

    params: hidden_size, num_heads, num_kv_heads, key_dim, value_dim, taps, query_scale, eps, decay_rank and gate_rank (random
    weights only), names (local tensor names; a convolution's is its projection's + conv_suffix), conv_suffix."""
    capturable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.nh, self.nkh = int(p["hidden_size"]), int(p["num_heads"]), int(p["num_kv_heads"])
        self.dk, self.dv, self.taps = int(p["key_dim"]), int(p["value_dim"]), int(p["taps"])
        self.q_scale, self.eps = float(p.get("query_scale", 1.0)), float(p["eps"])
        if self.nkh <= 0 or self.nh % self.nkh:
            raise ValueError(f"{self.nh} heads cannot share {self.nkh} query/key heads")
        if self.taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {self.taps}")
        limit = kernels.mixers.DELTA_MAX_DIM
        if not (0 < self.dk <= limit and 0 < self.dv <= limit):
            raise kernels.KernelError(f"delta rule: heads of {self.dk} key and {self.dv} value channels; the kernels take up to {limit}")
        self.a_rank, self.g_rank = int(p.get("decay_rank", 16)), int(p.get("gate_rank", 16))
        self.names = dict({k: k for k in ("q", "k", "v", "b", "A_log", "norm", "a1", "a2", "dt_bias", "g1", "g2", "o")}, **(p.get("names") or {}))
        self.conv_suffix = str(p.get("conv_suffix", ".conv"))
        self.channels = 2 * self.nkh * self.dk + self.nh * self.dv            # what the convolution runs over: q, k, v
        self.w_in = self.w_low = self.w_a2 = self.b_a2 = self.w_g2 = self.w_norm = self.w_o = self.conv = self.a_log = None

    def cache_users(self):
        return [(None, self.nh * self.dk * self.dv), (None, (self.taps - 1) * self.channels)]

    def tensors(self):
        n, D, K, V, A = self.names, self.hidden, self.nkh * self.dk, self.nh * self.dv, self.nh * self.dk
        t = {}
        for key, rows in (("q", K), ("k", K), ("v", V)):
            t[n[key]] = TensorDecl((rows, D))
            t[n[key] + self.conv_suffix] = TensorDecl((rows, self.taps), init="mean:0.25", use="vector")
        t.update({n["b"]: TensorDecl((self.nh, D)), n["A_log"]: TensorDecl((self.nh,), use="vector"),
                  n["norm"]: TensorDecl((self.dv,), init="one_plus_normal", use="vector"),
                  n["a1"]: TensorDecl((self.a_rank, D), free=(0,)), n["a2"]: TensorDecl((A, self.a_rank), free=(1,)),
                  n["dt_bias"]: TensorDecl((A,), use="vector"),
                  n["g1"]: TensorDecl((self.g_rank, D), free=(0,)), n["g2"]: TensorDecl((V, self.g_rank), free=(1,)),
                  n["o"]: TensorDecl((D, V))})
        return t

    def load(self, tensors):
        n = self.names
        self.a_rank, self.g_rank = int(tensors[n["a1"]].shape[0]), int(tensors[n["g1"]].shape[0])
        for first, second in (("a1", "a2"), ("g1", "g2")):
            if tensors[n[second]].shape[1] != tensors[n[first]].shape[0]:
                raise ValueError(f"the matrices {n[first]} and {n[second]} do not fit: {tuple(tensors[n[first]].shape)} and "
                                 f"{tuple(tensors[n[second]].shape)}")
        # (rows of zeros behind beta's keep the product's rows whole 16-byte pieces)
        self.w_in = _fuse([tensors[n[k]] for k in ("q", "k", "v", "b")] + [tensors[n["b"]].new_zeros((-(self.channels + self.nh) % 8, self.hidden))])
        self.conv = torch.cat([tensors[n[k] + self.conv_suffix].float() for k in ("q", "k", "v")], dim=0).t().contiguous()      # [taps, channels]
        # the second matrices read whole 16-byte pieces of the bottlenecks' rows: each bottleneck is padded with zero rows
        pad = lambda t, r: torch.cat([t, t.new_zeros((-r % 8, t.shape[1]))], dim=0)
        self.w_low = _fuse([pad(tensors[n["a1"]], self.a_rank), pad(tensors[n["g1"]], self.g_rank)])
        widen = lambda t, r: torch.cat([t, t.new_zeros((t.shape[0], -r % 8))], dim=1).contiguous()
        self.w_a2, self.w_g2 = widen(tensors[n["a2"]], self.a_rank), widen(tensors[n["g2"]], self.g_rank)
        self.b_a2 = tensors[n["dt_bias"]].float().contiguous()
        self.a_log = tensors[n["A_log"]].float().contiguous()
        self.w_norm = tensors[n["norm"]].contiguous()
        self.w_o = tensors[n["o"]].contiguous()

    def _heads(self, x, ctx, call):
        """[T, num_heads * value_dim], before the output projection."""
        A = self.w_a2.shape[1]
        proj = kernels.linear(x, self.w_in, out_dtype=torch.float32)                 # [T, q | k | v | beta's logits]
        low = kernels.linear(x, self.w_low)
        z = kernels.linear(low[:, :A], self.w_a2, self.b_a2, out_dtype=torch.float32)
        gate = kernels.linear(low[:, A:], self.w_g2)
        qkv, beta = kernels.delta_prep(proj, z, self.conv, self.a_log, ctx.state(call + 1) if self.taps > 1 else None, self.nkh, self.nh,
                                       self.dk, self.dv, self.q_scale, ctx, fast=x.dtype == torch.bfloat16)
        chunked = x.dtype == torch.bfloat16 and ctx.max_new >= kernels.mixers.DELTA_CHUNKED_FROM
        o = kernels.delta_scan(qkv, z, beta, ctx.state(call), ctx.seq_start, ctx.seq_slot, ctx.n_seqs, ctx.max_new, self.nkh, self.nh,
                               self.dk, self.dv, chunked=chunked)
        return kernels.gla_out(o, gate, self.w_norm, self.nh, self.dv, self.eps, x.dtype, gate_act="sigmoid")

    def forward(self, x, ctx, call):
        return kernels.linear(self._heads(x, ctx, call), self.w_o, out_dtype=torch.float32)

    def forward_into(self, x, ctx, call, residual):
        if not (x.dtype == torch.bfloat16 and self.w_o.dtype == torch.bfloat16
                and kernels.linear_into_ok(x.new_empty((x.shape[0], self.nh * self.dv)), self.w_o, None, residual)):
            return False
        kernels.linear_into(self._heads(x, ctx, call), self.w_o, None, residual)
        return True

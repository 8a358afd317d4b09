from __future__ import annotations

import torch

from .. import kernels
from .base import Mixer, TensorDecl, register_part


@register_part("mixer", "state_space")
class StateSpace(Mixer):
    """Structured state space duality (Mamba-2): a recurrent mixer with a matrix of memory per head, S [state, value_dim] in float32,
    and one decay per head and token.  With inner = num_heads * value_dim, N = state, G = groups:

        [z: inner | x: inner | B: G N | C: G N | dt: num_heads] = W_in h
        x, B, C side by side through a causal convolution of `taps` tokens per channel with a bias, and silu
        dt <- softplus(dt + dt_bias);  S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x      (head i reads group i / (heads / G))
        out = Wo (norm_groups parts of y * silu(z), each divided by its root mean square, times norm)

    The sequence's memory is two users of the cache's fixed-size state (zero when the sequence starts): the matrices S, and the
    convolution's last taps - 1 inputs.  Up to 256 tokens W_in is one product whose output stays float32; beyond, z, x, B and C
    leave a bfloat16 product and dt, in float32, one of its own.  Single tokens, short steps and the 32-bit path run token by token;
    longer steps in chunks (kernels.ssd_scan).  `out_scale` c: the part's output is multiplied by c (in the norm's float32 weight).

    params: hidden_size, num_heads, value_dim, state, groups, taps, norm_groups, eps, out_scale, names (local tensor names)."""
    capturable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.nh, self.dv = int(p["hidden_size"]), int(p["num_heads"]), int(p["value_dim"])
        self.n, self.groups, self.taps, self.norm_groups = int(p["state"]), int(p["groups"]), int(p["taps"]), int(p["norm_groups"])
        self.eps, self.out_scale = float(p["eps"]), float(p.get("out_scale", 1.0))
        self.inner = self.nh * self.dv
        if self.groups <= 0 or self.nh % self.groups:
            raise ValueError(f"{self.nh} heads cannot share {self.groups} groups")
        if self.norm_groups <= 0 or self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels cannot be normed in {self.norm_groups} equal parts")
        if self.taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {self.taps}")
        if not (0 < self.n <= kernels.mixers.SSD_MAX_STATE):
            raise kernels.KernelError(f"state space: {self.n} state rows a head; the kernels take up to {kernels.mixers.SSD_MAX_STATE}")
        self.names = dict({"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
                           "norm": "norm", "o": "o"}, **(p.get("names") or {}))
        self.channels = self.inner + 2 * self.groups * self.n              # what the convolution runs over: x, B, C
        self.dt_off = -(-(self.inner + self.channels) // 8) * 8            # dt's rows of the matrix as it is kept
        self.w_in = self.w_o = self.conv = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.w_norm = None

    def cache_users(self):
        return [(None, self.nh * self.n * self.dv), (None, (self.taps - 1) * self.channels)]

    def tensors(self):
        n = self.names
        return {n["in"]: TensorDecl((self.inner + self.channels + self.nh, self.hidden)),
                n["conv"]: TensorDecl((self.channels, self.taps), init="mean:0.25", use="vector"),
                n["conv_bias"]: TensorDecl((self.channels,), use="vector"), n["dt_bias"]: TensorDecl((self.nh,), use="vector"),
                n["A_log"]: TensorDecl((self.nh,), use="vector"), n["D"]: TensorDecl((self.nh,), init="one_plus_normal", use="vector"),
                n["norm"]: TensorDecl((self.inner,), init="one_plus_normal", use="vector"), n["o"]: TensorDecl((self.hidden, self.inner))}

    def load(self, tensors):
        t = lambda k: tensors[self.names[k]]
        w, rows = t("in"), self.inner + self.channels
        # zero rows bring dt's rows, and the end, to whole 16-byte pieces of the product's rows
        pad = lambda n: w.new_zeros((n, self.hidden))
        self.w_in = torch.cat([w[:rows], pad(self.dt_off - rows), w[rows:], pad(-self.nh % 8)], dim=0).contiguous()
        self.conv = t("conv").float().t().contiguous()                     # [taps, channels]
        self.conv_bias, self.dt_bias, self.a_log, self.skip = (t(k).float().contiguous() for k in ("conv_bias", "dt_bias", "A_log", "D"))
        self.w_norm = (t("norm").float() * self.out_scale).contiguous()
        self.w_o = t("o").contiguous()

    def _heads(self, x, ctx, call):
        """[T, inner], before the output projection."""
        if x.dtype == torch.bfloat16 and x.shape[0] > 256:
            proj = kernels.linear(x, self.w_in[:self.dt_off])
            dt = kernels.linear(x, self.w_in[self.dt_off:], out_dtype=torch.float32, plan=kernels.narrow_plan(x, self.w_in[self.dt_off:]))
        else:
            proj = kernels.linear(x, self.w_in, out_dtype=torch.float32)
            dt = proj[:, self.dt_off:]
        end = self.inner + self.channels
        xbc = kernels.short_conv(proj[:, self.inner:end], self.conv, self.conv_bias, ctx.state(call + 1) if self.taps > 1 else None, ctx,
                                 act="silu", out_dtype=x.dtype)
        chunked = x.dtype == torch.bfloat16 and ctx.max_new >= kernels.mixers.SSD_CHUNKED_FROM
        y = kernels.ssd_scan(xbc, dt[:, :self.nh], self.dt_bias, self.a_log, self.skip, ctx.state(call), ctx.seq_start, ctx.seq_slot,
                             ctx.n_seqs, ctx.max_new, self.nh, self.dv, self.n, self.groups, chunked=chunked)
        return kernels.gated_group_norm(y, proj[:, :self.inner], self.w_norm, self.norm_groups, self.eps, x.dtype)

    def forward(self, x, ctx, call):
        return kernels.linear_f32(self._heads(x, ctx, call), self.w_o)

    def forward_into(self, x, ctx, call, residual):
        if not (x.dtype == torch.bfloat16 and self.w_o.dtype == torch.bfloat16
                and kernels.linear_into_ok(x.new_empty((x.shape[0], self.inner)), self.w_o, None, residual)):
            return False
        kernels.linear_into(self._heads(x, ctx, call), self.w_o, None, residual)
        return True

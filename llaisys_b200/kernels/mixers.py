"""Python faces of the kernels of the recurrent and the latent mixers (csrc/gla.cu, csrc/delta.cu, csrc/shortconv.cu, csrc/ssd.cu, csrc/headout.cu,
csrc/latent.cu, and the CUDA-core
attention kernel of csrc/attention_simt.cu run over a cache of latent rows)."""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_void_p
from typing import Optional

import torch

from ..csrc.build import load_module
from .ops import DT, KernelError, _AttnParams, _attn_lib, _check, _dt, _fn, _need_cuda, _ptr, _sm_count, _stream, _tc_resources


class _GlaParams(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("k", c_void_p), ("v", c_void_p), ("row_stride", c_int), ("z", c_void_p), ("z_stride", c_int),
                ("state", c_void_p), ("seq_start", c_void_p), ("seq_slot", c_void_p), ("out", c_void_p), ("H", c_int),
                ("dk", c_int), ("dv", c_int), ("q_scale", c_float), ("inv_tau", c_float), ("z_is_decay", c_int),
                ("head_decay", c_void_p), ("act", c_int)]


GLA_MAX_KEY_DIM = 256


def gla_scan(proj: torch.Tensor, H: int, dk: int, dv: int, z: Optional[torch.Tensor], state: torch.Tensor, seq_start: torch.Tensor,
             seq_slot: torch.Tensor, n_seqs: int, q_scale: float, decay_root: float, head_decay: Optional[torch.Tensor] = None,
             act: Optional[str] = None) -> torch.Tensor:
    """The gated-linear-attention recurrence over the new tokens of every sequence: proj [T, >= 2 H dk + H dv] holds the
    heads' queries, then keys, then values; z [T, H dk] (float32) the decay logits; state [slots, H dk dv] (float32) is
    read at row seq_slot[b] and left holding the state after the step.  Returns o [T, H dv] in float32.  For more than
    64 tokens the decays are formed by a pass of their own over z (in place), once per token and channel.
    head_decay (float32 [H]) instead of z: one constant decay per head, S <- decay_h S + k v^T.  act "silu": q, k and v
    pass through silu (in float32) on their way into the recurrence."""
    _need_cuda(proj, z, state, head_decay)
    assert (z is None) != (head_decay is None)
    assert z is None or (z.dtype == torch.float32 and z.stride(1) == 1)
    assert head_decay is None or (head_decay.dtype == torch.float32 and head_decay.numel() == H and head_decay.is_contiguous())
    assert state.dtype == torch.float32 and state.is_contiguous()
    assert proj.stride(1) == 1 and state.shape[1] == H * dk * dv
    if dk > GLA_MAX_KEY_DIM:
        raise KernelError(f"gated linear attention: {dk} key channels a head; the kernel takes up to {GLA_MAX_KEY_DIM}")
    T = proj.shape[0]
    out = torch.empty((T, H * dv), dtype=torch.float32, device=proj.device)
    p = _GlaParams()
    es = proj.element_size()
    p.q, p.k, p.v = proj.data_ptr(), proj.data_ptr() + H * dk * es, proj.data_ptr() + 2 * H * dk * es
    p.row_stride, p.z, p.z_stride = proj.stride(0), _ptr(z), z.stride(0) if z is not None else 0
    p.head_decay, p.act = _ptr(head_decay), {None: 0, "silu": 1}[act]
    p.state, p.seq_start, p.seq_slot, p.out = state.data_ptr(), seq_start.data_ptr(), seq_slot.data_ptr(), out.data_ptr()
    p.H, p.dk, p.dv, p.q_scale, p.inv_tau = H, dk, dv, q_scale, 1.0 / decay_root
    if z is not None and T > 64 and z.is_contiguous():
        g = _fn(load_module("gla.cu"), "llb_gla_decay", [c_void_p, ctypes.c_longlong, c_float, c_void_p])
        _check(g(_ptr(z), z.numel(), 1.0 / decay_root, _stream()), "gated linear attention (decays)")
        p.z_is_decay = 1
    f = _fn(load_module("gla.cu"), "llb_gla_scan", [_GlaParams, c_int, c_int, c_int, c_void_p])
    _check(f(p, _dt(proj), n_seqs, _sm_count(proj.device), _stream()), "gated linear attention (recurrence)")
    return out


SCAN_CHUNK = 64               # tokens of a chunk of a long step of the constant-decay recurrence
SCAN_CHUNKED_FROM = 256       # steps whose longest sequence brings at least this many tokens run chunk by chunk


def scan_chunks(n_new, device, chunk: int = SCAN_CHUNK):
    """The chunks of a step whose sequences bring n_new[b] tokens: int32 device tensors chunk_start [NC + 1] (first packed
    token of every chunk), chunk_len [NC], seq_chunk0 [B + 1] (first chunk of every sequence), chunk_row [NC] (0 .. NC - 1)."""
    starts, lens, seq0, at = [], [], [0], 0
    for n in n_new:
        for c0 in range(0, n, chunk):
            starts.append(at + c0)
            lens.append(min(chunk, n - c0))
        at += n
        seq0.append(len(starts))
    starts.append(at)
    flat = torch.tensor(starts + lens + seq0 + list(range(len(lens))), dtype=torch.int32).to(device)
    nc, b = len(lens), len(n_new)
    return flat[:nc + 1], flat[nc + 1:2 * nc + 1], flat[2 * nc + 1:2 * nc + 2 + b], flat[2 * nc + 2 + b:]


def gla_scan_chunked(proj: torch.Tensor, H: int, dk: int, dv: int, state: torch.Tensor, seq_slot: torch.Tensor, n_seqs: int,
                     head_decay: torch.Tensor, chunks, act: Optional[str] = None) -> torch.Tensor:
    """The constant-decay recurrence (gla_scan with head_decay) of a long step, its chunks side by side: the recurrence over
    every chunk from a zero state, one pass that turns the chunks' local states into the states they start with (and
    leaves the sequences' states as the step ends them), and the recurrence over every chunk again.  chunks: scan_chunks()
    of the step.  Returns o [T, H dv] in float32; differs from the token-by-token walk by float32 rounding only."""
    chunk_start, chunk_len, seq_chunk0, chunk_row = chunks
    nc = chunk_len.numel()
    n_state = H * dk * dv
    tmp = torch.zeros((nc, n_state), dtype=torch.float32, device=proj.device)
    gla_scan(proj, H, dk, dv, None, tmp, chunk_start, chunk_row, nc, 1.0, 1.0, head_decay=head_decay, act=act)
    f = _fn(load_module("gla.cu"), "llb_gla_chunk_prefix", [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                                           c_int, c_void_p])
    _check(f(_ptr(tmp), _ptr(state), _ptr(seq_chunk0), _ptr(chunk_len), _ptr(seq_slot), _ptr(head_decay), dk * dv, n_state, n_seqs,
             _stream()), "constant-decay recurrence (chunks' starting states)")
    return gla_scan(proj, H, dk, dv, None, tmp, chunk_start, chunk_row, nc, 1.0, 1.0, head_decay=head_decay, act=act)


def gla_out(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, H: int, dv: int, eps: float,
            out_dtype: torch.dtype, gate_act: str = "silu") -> torch.Tensor:
    """[T, H dv]: every head's o (float32) RMS-normed over its dv channels with `weight` [dv], times silu(gate) (gate a
    [T, H dv] view with any row stride, in the output's dtype)."""
    _need_cuda(o, gate, weight)
    T = o.shape[0]
    assert o.dtype == torch.float32 and o.is_contiguous() and gate.dtype == out_dtype and gate.stride(1) == 1
    out = torch.empty((T, H * dv), dtype=out_dtype, device=o.device)
    f = _fn(load_module("headout.cu"), "llb_gla_out", [c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_int,
                                                  c_int, c_float, c_int, c_void_p])
    _check(f(_ptr(o), _ptr(gate), gate.stride(0), _ptr(weight), _dt(weight), _ptr(out), DT[out_dtype], T, H, dv, eps,
             {"silu": 0, "sigmoid": 1}[gate_act], _stream()),
           "gated linear attention (head norm and gate)")
    return out


class _DeltaPrepParams(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ld", c_int), ("z", c_void_p), ("conv_w", c_void_p), ("a_log", c_void_p), ("conv_state", c_void_p),
                ("seq_start", c_void_p), ("seq_slot", c_void_p), ("out", c_void_p), ("beta", c_void_p),
                ("G", c_int), ("H", c_int), ("dk", c_int), ("dv", c_int), ("taps", c_int), ("q_scale", c_float),
                ("fast", c_int), ("vec", c_int)]


DELTA_MAX_DIM = 256           # key and value channels of a head


def delta_prep(proj: torch.Tensor, z: torch.Tensor, conv_w: torch.Tensor, a_log: torch.Tensor, conv_state: Optional[torch.Tensor],
               G: int, H: int, dk: int, dv: int, q_scale: float, ctx, fast: bool = False):
    """What enters the delta rule, from proj [T, >= C + H] (float32; C = 2 G dk + H dv: q, k of G heads and v of H heads, then
    one step-size logit per head) and the decays' logits z [T, H dk] (float32, contiguous, replaced in place by the decays
    exp(-exp(a_log) softplus(z))): (rows [T, C], beta [T, H]) with the short causal convolution (conv_w float32 [taps, C],
    the last row for the current token) and silu applied, every head's q and k made unit vectors (q times q_scale) and
    beta = sigmoid(logit).  conv_state (float32 [slots, (taps - 1) C], oldest input first; None with one tap) holds each
    sequence's last inputs and is brought up to date.  fast: silu by the special-function unit (for the bfloat16 path)."""
    _need_cuda(proj, z, conv_w, a_log, conv_state)
    T = proj.shape[0]
    C, taps = 2 * G * dk + H * dv, conv_w.shape[0]
    assert proj.dtype == z.dtype == conv_w.dtype == a_log.dtype == torch.float32 and proj.stride(1) == 1 and proj.shape[1] >= C + H
    assert z.is_contiguous() and z.shape == (T, H * dk) and conv_w.is_contiguous() and conv_w.shape[1] == C and a_log.numel() == H
    assert taps == 1 or (conv_state.dtype == torch.float32 and conv_state.is_contiguous() and conv_state.shape[1] == (taps - 1) * C)
    out = torch.empty((T, C), dtype=torch.float32, device=proj.device)
    beta = torch.empty((T, H), dtype=torch.float32, device=proj.device)
    p = _DeltaPrepParams()
    p.proj, p.ld, p.z, p.conv_w, p.a_log, p.conv_state = proj.data_ptr(), proj.stride(0), z.data_ptr(), conv_w.data_ptr(), a_log.data_ptr(), _ptr(conv_state)
    p.seq_start, p.seq_slot, p.out, p.beta = ctx.seq_start.data_ptr(), ctx.seq_slot.data_ptr(), out.data_ptr(), beta.data_ptr()
    p.G, p.H, p.dk, p.dv, p.taps, p.q_scale, p.fast = G, H, dk, dv, taps, q_scale, int(fast)
    f = _fn(load_module("delta.cu"), "llb_delta_prep", [_DeltaPrepParams, c_int, c_int, c_void_p])
    _check(f(p, ctx.n_seqs, ctx.max_new, _stream()), "delta rule (convolution, unit vectors, decays)")
    return out, beta


class _DeltaScanParams(ctypes.Structure):
    _fields_ = [("qkv", c_void_p), ("g", c_void_p), ("beta", c_void_p), ("state", c_void_p), ("seq_start", c_void_p), ("seq_slot", c_void_p),
                ("out", c_void_p), ("G", c_int), ("H", c_int), ("dk", c_int), ("dv", c_int)]


class _DeltaChunkParams(ctypes.Structure):
    _fields_ = [("qkv", c_void_p), ("g", c_void_p), ("beta", c_void_p), ("state", c_void_p), ("seq_start", c_void_p), ("seq_slot", c_void_p),
                ("out", c_void_p), ("rec", c_void_p), ("err", c_void_p), ("G", c_int), ("H", c_int), ("dk", c_int), ("dv", c_int), ("cb", c_int)]


DELTA_CHUNKED_FROM = 32       # steps whose longest sequence brings at least this many tokens run in chunks


def delta_scan(qkv: torch.Tensor, g: torch.Tensor, beta: torch.Tensor, state: torch.Tensor, seq_start: torch.Tensor, seq_slot: torch.Tensor,
               n_seqs: int, max_new: int, G: int, H: int, dk: int, dv: int, chunked: bool = False) -> torch.Tensor:
    """The gated delta rule over the new tokens of every sequence: qkv [T, 2 G dk + H dv], g [T, H dk] (decays) and
    beta [T, H], all float32; state [slots, H dk dv] (float32) is read at row seq_slot[b] and left holding the state after
    the step.  Returns o [T, H dv] in float32.  chunked: chunks of 16 tokens on the tensor cores (float32 operands split
    into two TF32 numbers each, float32 sums) instead of token by token on the CUDA cores."""
    _need_cuda(qkv, g, beta, state)
    T = qkv.shape[0]
    assert qkv.dtype == g.dtype == beta.dtype == state.dtype == torch.float32
    assert qkv.is_contiguous() and g.is_contiguous() and beta.is_contiguous() and state.is_contiguous()
    assert qkv.shape[1] == 2 * G * dk + H * dv and g.shape == (T, H * dk) and beta.shape == (T, H) and state.shape[1] == H * dk * dv
    out = torch.empty((T, H * dv), dtype=torch.float32, device=qkv.device)
    p = _DeltaChunkParams() if chunked else _DeltaScanParams()
    p.qkv, p.g, p.beta, p.state, p.out = qkv.data_ptr(), g.data_ptr(), beta.data_ptr(), state.data_ptr(), out.data_ptr()
    p.seq_start, p.seq_slot, p.G, p.H, p.dk, p.dv = seq_start.data_ptr(), seq_slot.data_ptr(), G, H, dk, dv
    lib = load_module("delta.cu")
    if not chunked:
        f = _fn(lib, "llb_delta_scan", [_DeltaScanParams, c_int, c_int, c_void_p])
        _check(f(p, n_seqs, _sm_count(qkv.device), _stream()), "delta rule (recurrence)")
        return out
    size = lib.llb_delta_scratch
    size.argtypes, size.restype = [c_int, c_int, c_int, c_int, c_int], ctypes.c_longlong
    rec = torch.empty(int(size(T, n_seqs, H, dk, dv)), dtype=torch.float32, device=qkv.device)
    p.rec, p.err = rec.data_ptr(), _tc_resources(qkv.device)[2].data_ptr()
    f = _fn(lib, "llb_delta_chunked", [_DeltaChunkParams, c_int, c_int, c_int, c_void_p])
    _check(f(p, n_seqs, max_new, _sm_count(qkv.device), _stream()), "delta rule (recurrence in chunks)", 2)
    del rec
    return out


class _ShortConvParams(ctypes.Structure):
    _fields_ = [("x", c_void_p), ("ld", c_int), ("w", c_void_p), ("bias", c_void_p), ("state", c_void_p), ("seq_start", c_void_p),
                ("seq_slot", c_void_p), ("C", c_int), ("taps", c_int)]


class _ConvHeadsParams(ctypes.Structure):
    _fields_ = [("conv", _ShortConvParams), ("out", c_void_p), ("ldo", c_int), ("n_q", c_int), ("n_k", c_int), ("d", c_int), ("rot", c_int),
                ("v_mult", c_float), ("cos_t", c_void_p), ("sin_t", c_void_p), ("table_rows", c_int), ("tok_pos", c_void_p),
                ("append", c_int), ("seq_len_before", c_void_p), ("kpool", c_void_p), ("vpool", c_void_p), ("page_table", c_void_p),
                ("table_stride", c_int), ("ring", c_int), ("pinned", c_int), ("err", c_void_p)]


def _conv_params(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: Optional[torch.Tensor], ctx) -> _ShortConvParams:
    _need_cuda(x, w, bias, state)
    taps, C = w.shape
    assert x.stride(1) == 1 and x.shape[1] == C and w.dtype == torch.float32 and w.is_contiguous()
    assert bias is None or (bias.dtype == torch.float32 and bias.numel() == C and bias.is_contiguous())
    assert taps == 1 or (state.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == (taps - 1) * C)
    p = _ShortConvParams()
    p.x, p.ld, p.w, p.bias, p.state = x.data_ptr(), x.stride(0), w.data_ptr(), _ptr(bias), _ptr(state) if taps > 1 else None
    p.seq_start, p.seq_slot, p.C, p.taps = ctx.seq_start.data_ptr(), ctx.seq_slot.data_ptr(), C, taps
    return p


def short_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: Optional[torch.Tensor], ctx, act: Optional[str] = None,
               out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """The causal convolution of every channel of x [T, C] (row stride free) over its sequence's tokens, plus bias (float32 [C] or
    None), then act (None or "silu"): [T, C] in out_dtype.  w float32 [taps, C], the last row for the current token; state (float32
    [slots, (taps - 1) C], oldest input first; None with one tap) holds each sequence's last inputs and is brought up to date."""
    p = _conv_params(x, w, bias, state, ctx)
    out = torch.empty((x.shape[0], p.C), dtype=out_dtype or x.dtype, device=x.device)
    f = _fn(load_module("shortconv.cu"), "llb_short_conv", [_ShortConvParams, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _check(f(p, _dt(x), _ptr(out), _dt(out), out.stride(0), {None: 0, "silu": 1}[act], ctx.n_seqs, ctx.max_new, _stream()), "short convolution")
    return out


def conv_heads(x: torch.Tensor, n_q: int, n_k: int, d: int, w: torch.Tensor, state: Optional[torch.Tensor], ctx, tables=None,
               v_mult: float = 1.0, append: Optional[dict] = None) -> torch.Tensor:
    """From the projections x [T, (n_q + n_k) d] of query and key heads, each channel through a causal convolution (w, state as for
    short_conv): packed [T, (n_q + 2 n_k) d] with the queries and keys, their first `dims` dimensions rotated in pairs
    (i, i + dims / 2) by tables = (cos, sin, dims), and the values: the convolved keys before the rotation, times v_mult.  append =
    dict(seq_len_before, kpool, vpool, page_table, ring, pinned): the keys and values also go into the paged cache."""
    T = x.shape[0]
    p = _ConvHeadsParams()
    p.conv = _conv_params(x, w, None, state, ctx)
    out = torch.empty((T, (n_q + 2 * n_k) * d), dtype=x.dtype, device=x.device)
    p.out, p.ldo, p.n_q, p.n_k, p.d, p.v_mult = out.data_ptr(), out.stride(0), n_q, n_k, d, v_mult
    if tables is not None:
        cos, sin, dims = tables
        assert cos.dtype == sin.dtype == torch.float32 and cos.shape[1] == dims // 2 and cos.is_contiguous() and sin.is_contiguous()
        p.rot, p.cos_t, p.sin_t, p.table_rows = dims, cos.data_ptr(), sin.data_ptr(), cos.shape[0]
    p.tok_pos, p.err = ctx.tok_pos.data_ptr(), ctx.err.data_ptr()
    if append is not None:
        a = append
        assert a["kpool"].dtype == a["vpool"].dtype == x.dtype
        p.append, p.seq_len_before, p.kpool, p.vpool = 1, a["seq_len_before"].data_ptr(), a["kpool"].data_ptr(), a["vpool"].data_ptr()
        p.page_table, p.table_stride, p.ring, p.pinned = a["page_table"].data_ptr(), a["page_table"].shape[1], a["ring"], a.get("pinned", 0)
    f = _fn(load_module("shortconv.cu"), "llb_conv_heads", [_ConvHeadsParams, c_int, c_int, c_int, c_void_p])
    _check(f(p, _dt(x), ctx.n_seqs, ctx.max_new, _stream()), "short convolution, rotation and cache append of heads")
    return out


class _SsdParams(ctypes.Structure):
    _fields_ = [("xbc", c_void_p), ("ld", c_int), ("dt", c_void_p), ("dt_ld", c_int), ("dt_bias", c_void_p), ("a_log", c_void_p),
                ("skip", c_void_p), ("state", c_void_p), ("seq_start", c_void_p), ("seq_slot", c_void_p), ("out", c_void_p),
                ("H", c_int), ("P", c_int), ("N", c_int), ("G", c_int), ("rec", c_void_p), ("decay", c_void_p),
                ("sums", c_void_p)]


SSD_MAX_STATE = 256           # rows of a head's state
SSD_CHUNKED_FROM = 32         # steps whose longest sequence brings at least this many tokens run in chunks


def ssd_scan(xbc: torch.Tensor, dt: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor, state: torch.Tensor,
             seq_start: torch.Tensor, seq_slot: torch.Tensor, n_seqs: int, max_new: int, H: int, P: int, N: int, G: int,
             chunked: bool = False) -> torch.Tensor:
    """The state-space recurrence over the new tokens of every sequence: xbc [T, H P + 2 G N] holds x (H heads of P), B and C (G
    groups of N); dt (float32 [T, H], row stride free) the logits of the step sizes softplus(dt + dt_bias); S <- exp(-exp(a_log)
    step) S + step B x^T, y = S^T C + skip x; state [slots, H N P] (float32) is read at row seq_slot[b] and left holding the state
    after the step.  Returns y [T, H P] in float32.  chunked (bfloat16 xbc): chunks of 64 tokens on the tensor cores instead of token
    by token on the CUDA cores."""
    _need_cuda(xbc, dt, dt_bias, a_log, skip, state)
    T = xbc.shape[0]
    assert xbc.stride(1) == 1 and xbc.shape[1] == H * P + 2 * G * N and dt.dtype == torch.float32 and dt.shape == (T, H) and dt.stride(1) == 1
    for v in (dt_bias, a_log, skip):
        assert v.dtype == torch.float32 and v.numel() == H and v.is_contiguous()
    assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == H * N * P
    if N > SSD_MAX_STATE:
        raise KernelError(f"state space: {N} state rows a head; the kernels take up to {SSD_MAX_STATE}")
    out = torch.empty((T, H * P), dtype=torch.float32, device=xbc.device)
    p = _SsdParams()
    p.xbc, p.ld, p.dt, p.dt_ld = xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), dt.stride(0)
    p.dt_bias, p.a_log, p.skip, p.state = dt_bias.data_ptr(), a_log.data_ptr(), skip.data_ptr(), state.data_ptr()
    p.seq_start, p.seq_slot, p.out, p.H, p.P, p.N, p.G = seq_start.data_ptr(), seq_slot.data_ptr(), out.data_ptr(), H, P, N, G
    lib = load_module("ssd.cu")
    if not chunked:
        f = _fn(lib, "llb_ssd_scan", [_SsdParams, c_int, c_int, c_void_p])
        _check(f(p, _dt(xbc), n_seqs, _stream()), "state space (recurrence)")
        return out
    assert xbc.dtype == torch.bfloat16
    chunks = _fn(lib, "llb_ssd_chunks", [c_int, c_int])(T, n_seqs)
    rec = torch.empty((chunks, H * N * P), dtype=torch.float32, device=xbc.device)
    small = torch.empty((chunks * H * 129,), dtype=torch.float32, device=xbc.device)
    p.rec, p.sums, p.decay = rec.data_ptr(), small.data_ptr(), small[chunks * H * 128:].data_ptr()
    f = _fn(lib, "llb_ssd_chunked", [_SsdParams, c_int, c_int, c_void_p])
    _check(f(p, n_seqs, max_new, _stream()), "state space (recurrence in chunks)", 3)
    del rec, small
    return out


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, groups: int, eps: float, out_dtype: torch.dtype) -> torch.Tensor:
    """[T, C]: g = y * silu(z) (y float32, z a view with any row stride), each of `groups` equal parts of the row divided by its own
    sqrt(mean(g^2) + eps), times weight (float32 [C])."""
    _need_cuda(y, z, weight)
    T, C = y.shape
    assert y.dtype == torch.float32 and y.is_contiguous() and z.shape == (T, C) and z.stride(1) == 1
    assert weight.dtype == torch.float32 and weight.numel() == C and weight.is_contiguous() and groups > 0 and C % groups == 0
    out = torch.empty((T, C), dtype=out_dtype, device=y.device)
    f = _fn(load_module("ssd.cu"), "llb_gated_group_norm", [c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                                            c_float, c_void_p])
    _check(f(_ptr(y), _ptr(z), _dt(z), z.stride(0), _ptr(weight), _ptr(out), DT[out_dtype], T, groups, C // groups, eps, _stream()),
           "gate and norm in parts")
    return out


class _MinGruParams(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ld", c_int), ("a_off", c_int), ("u_off", c_int), ("g_off", c_int), ("width", c_int),
                ("state", c_void_p), ("seq_start", c_void_p), ("seq_slot", c_void_p), ("out", c_void_p), ("chunk_a", c_void_p),
                ("chunk_b", c_void_p), ("chunk", c_int), ("n_chunks", c_int)]


MINGRU_CHUNK = 64            # tokens of a chunk of a long step (256 beyond 4,096 tokens a sequence)


def mingru(proj: torch.Tensor, width: int, state: torch.Tensor, seq_start: torch.Tensor, seq_slot: torch.Tensor, n_seqs: int,
           max_new: int, out_dtype: torch.dtype, offsets=None) -> torch.Tensor:
    """The minGRU recurrence over the new tokens of every sequence: proj [T, >= 3 width] holds the gate logits, the
    candidate inputs and the output gate (`offsets` = their first columns, default 0, width, 2 width), biases included;
    state [slots, width] (float32) is read at row seq_slot[b] and left holding the state after the step.  Returns
    y [T, width] = state_t * silu(output gate) in out_dtype.  Steps of more than one chunk of tokens a sequence are cut
    into chunks that run side by side (three launches instead of one)."""
    _need_cuda(proj, state)
    assert proj.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == width
    T = proj.shape[0]
    a_off, u_off, g_off = offsets or (0, width, 2 * width)
    out = torch.empty((T, width), dtype=out_dtype, device=proj.device)
    p = _MinGruParams()
    p.proj, p.ld, p.a_off, p.u_off, p.g_off, p.width = proj.data_ptr(), proj.stride(0), a_off, u_off, g_off, width
    p.state, p.seq_start, p.seq_slot, p.out = state.data_ptr(), seq_start.data_ptr(), seq_slot.data_ptr(), out.data_ptr()
    p.chunk = MINGRU_CHUNK if max_new <= 4096 else 256
    p.n_chunks = -(-max_new // p.chunk)
    scratch, launches = None, 1
    if p.n_chunks > 1:
        scratch = torch.empty((2, n_seqs, p.n_chunks, width), dtype=torch.float32, device=proj.device)
        p.chunk_a, p.chunk_b = scratch[0].data_ptr(), scratch[1].data_ptr()
        launches = 3
    f = _fn(load_module("mingru.cu"), "llb_mingru", [_MinGruParams, c_int, c_int, c_int, c_void_p])
    _check(f(p, _dt(proj), DT[out_dtype], n_seqs, _stream()), "minGRU recurrence", launches)
    del scratch
    return out


class _LatentPrepParams(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("row_stride", c_int), ("q_off", c_int), ("q_rank", c_int), ("kv_off", c_int),
                ("kv_rank", c_int), ("kr_off", c_int), ("rope_dim", c_int), ("rot", c_int), ("wq", c_void_p), ("wkv", c_void_p),
                ("eps", c_float), ("cos_t", c_void_p), ("sin_t", c_void_p), ("table_rows", c_int), ("tok_pos", c_void_p),
                ("q_out", c_void_p), ("kv_out", c_void_p), ("append", c_int), ("tok_seq", c_void_p), ("seq_start", c_void_p),
                ("seq_len_before", c_void_p), ("pool", c_void_p), ("page_table", c_void_p), ("table_stride", c_int),
                ("ring", c_int), ("pinned", c_int), ("err", c_void_p), ("halves", c_int)]


def latent_prep(proj: torch.Tensor, q_rank: int, kv_rank: int, rope_dim: int, wq: Optional[torch.Tensor], wkv: Optional[torch.Tensor],
                eps: float, tables, tok_pos: torch.Tensor, err: torch.Tensor, append: Optional[dict] = None, halves: bool = False,
                kv_off: Optional[int] = None):
    """From the fused down projections proj [T, q_rank (+ kv_rank + rope_dim) ...]: the RMS-normed query latent
    [T, q_rank] and, when the layer projects its own (wkv given), the rows [normed latent | rotated shared key part]
    [T, kv_rank + rope_dim]; tables = (cos, sin, rotated dims) or None.  append = dict(tok_seq, seq_start,
    seq_len_before, pool, page_table, ring, pinned) also writes those rows into the paged cache.  halves: the rotated
    pairs are (i, i + dims / 2) instead of (2i, 2i + 1).  q_rank 0 (wq None): the layer has no query latent; kv_off then
    says where the key/value latent's columns start (default: after the query latent)."""
    _need_cuda(proj, wq, wkv, tok_pos)
    T = proj.shape[0]
    assert proj.stride(1) == 1 and tok_pos.numel() == T
    own = wkv is not None
    assert (q_rank > 0) == (wq is not None) and (own or q_rank > 0)
    q_out = torch.empty((T, q_rank), dtype=proj.dtype, device=proj.device) if q_rank > 0 else None
    kv_out = torch.empty((T, kv_rank + rope_dim), dtype=proj.dtype, device=proj.device) if own else None
    p = _LatentPrepParams()
    p.proj, p.row_stride, p.q_off, p.q_rank = proj.data_ptr(), proj.stride(0), 0, q_rank
    off = q_rank if kv_off is None else int(kv_off)
    p.kv_off, p.kv_rank, p.kr_off, p.rope_dim = off, kv_rank if own else 0, off + kv_rank, rope_dim
    p.wq, p.wkv, p.eps, p.halves = _ptr(wq), _ptr(wkv), eps, int(halves)
    if own and wq is not None and wkv.dtype != wq.dtype:
        raise KernelError("latent_prep: the two norm weights must have one dtype")
    if tables is not None and own:
        cos, sin, rot = tables
        p.cos_t, p.sin_t, p.table_rows, p.rot = cos.data_ptr(), sin.data_ptr(), cos.shape[0], rot
    p.tok_pos, p.q_out, p.kv_out, p.err = tok_pos.data_ptr(), _ptr(q_out), _ptr(kv_out), err.data_ptr()
    if append is not None and own:
        a = append
        p.append, p.tok_seq, p.seq_start, p.seq_len_before = 1, a["tok_seq"].data_ptr(), a["seq_start"].data_ptr(), a["seq_len_before"].data_ptr()
        p.pool, p.page_table, p.table_stride = a["pool"].data_ptr(), a["page_table"].data_ptr(), a["page_table"].shape[1]
        p.ring, p.pinned = a["ring"], a.get("pinned", 0)
    f = _fn(load_module("latent.cu"), "llb_latent_prep", [_LatentPrepParams, c_int, c_int, c_int, c_void_p])
    _check(f(p, _dt(proj), _dt(wq if wq is not None else wkv), T, _stream()), "latent attention (norms, key rotation, cache rows)")
    return q_out, kv_out


def latent_append(rows: torch.Tensor, tok_pos: torch.Tensor, append: dict) -> None:
    """rows [T, width] into the tokens' rows of the paged cache (a pool of one key head of `width` elements)."""
    _need_cuda(rows, tok_pos)
    assert rows.is_contiguous()
    a = append
    f = _fn(load_module("latent.cu"), "llb_latent_append", [c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                                                            c_void_p, c_void_p, c_int, c_int, c_int, c_void_p])
    _check(f(_ptr(rows), _dt(rows), rows.shape[0], rows.shape[1], _ptr(tok_pos), _ptr(a["tok_seq"]), _ptr(a["seq_start"]),
             _ptr(a["seq_len_before"]), _ptr(a["pool"]), _ptr(a["page_table"]), a["page_table"].shape[1], a["ring"],
             a.get("pinned", 0), _stream()), "latent attention (cache append)")


class _HeadMatmulParams(ctypes.Structure):
    _fields_ = [("x", c_void_p), ("x_stride", c_int), ("x_head", c_int), ("m", c_void_p), ("y", c_void_p), ("y_stride", c_int),
                ("y_head", c_int), ("T", c_int), ("H", c_int), ("n_in", c_int), ("n_out", c_int), ("tail", c_int), ("rot", c_int),
                ("cos_t", c_void_p), ("sin_t", c_void_p), ("table_rows", c_int), ("tok_pos", c_void_p), ("gate", c_void_p),
                ("gate_stride", c_int), ("err", c_void_p), ("halves", c_int), ("gate_elems", c_int)]


def head_matmul(x: torch.Tensor, m: torch.Tensor, *, tail: int = 0, tables=None, tok_pos=None, gate: Optional[torch.Tensor] = None,
                err: Optional[torch.Tensor] = None, halves: bool = False, gate_elems: bool = False) -> torch.Tensor:
    """y[t, h, :n_out] = x[t, h, :n_in] m[h] for x [T, H (n_in + tail)] and m [H, n_in, n_out], float32 accumulation; the
    `tail` elements after a head's inputs follow its outputs in y [T, H (n_out + tail)], the first `rot` of them rotated in
    pairs (2i, 2i+1) by tables = (cos, sin, rot) at the tokens' positions; with gate ([T, >= H] view) every head's
    outputs are multiplied by sigmoid(gate[t, h]), or, with gate_elems, output element i of head h by
    sigmoid(gate[t, h n_out + i]) (gate a [T, >= H n_out] view).  halves: the rotated pairs are (i, i + rot / 2)."""
    _need_cuda(x, m, gate, tok_pos)
    T = x.shape[0]
    H, n_in, n_out = m.shape
    assert x.stride(1) == 1 and m.is_contiguous() and m.dtype == x.dtype and x.shape[1] == H * (n_in + tail)
    y = torch.empty((T, H * (n_out + tail)), dtype=x.dtype, device=x.device)
    p = _HeadMatmulParams()
    p.x, p.x_stride, p.x_head, p.m = x.data_ptr(), x.stride(0), n_in + tail, m.data_ptr()
    p.y, p.y_stride, p.y_head = y.data_ptr(), y.stride(0), n_out + tail
    p.T, p.H, p.n_in, p.n_out, p.tail = T, H, n_in, n_out, tail
    p.halves, p.gate_elems = int(halves), int(gate_elems)
    if tail and tables is not None:
        cos, sin, rot = tables
        if tok_pos is None or err is None:
            raise KernelError("head_matmul: a rotated tail needs the tokens' positions and an error word")
        p.cos_t, p.sin_t, p.table_rows, p.rot, p.tok_pos, p.err = cos.data_ptr(), sin.data_ptr(), cos.shape[0], rot, tok_pos.data_ptr(), err.data_ptr()
    if gate is not None:
        assert gate.dtype == x.dtype and gate.stride(1) == 1
        p.gate, p.gate_stride = gate.data_ptr(), gate.stride(0)
    f = _fn(load_module("latent.cu"), "llb_head_matmul", [_HeadMatmulParams, c_int, c_void_p])
    _check(f(p, _dt(x), _stream()), "per-head matrix product")
    return y


def rope_pairs_(x: torch.Tensor, H: int, head: int, off: int, tables, tok_pos: torch.Tensor, err: torch.Tensor,
                halves: bool = False) -> None:
    """In place on x [T, >= H head] (row stride free): of every head's elements from `off` on, the pairs (2i, 2i+1)
    (with halves: (i, i + rot / 2)), i < rot / 2, are rotated by tables = (cos, sin, rot) at the tokens' positions."""
    _need_cuda(x, tok_pos)
    if tables is None:
        return
    cos, sin, rot = tables
    assert x.stride(1) == 1 and off + rot <= head
    f = _fn(load_module("latent.cu"), "llb_rope_pairs", [c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p,
                                                         c_int, c_void_p, c_void_p, c_int, c_void_p])
    _check(f(_ptr(x), _dt(x), x.shape[0], x.stride(0), H, head, off, rot, _ptr(cos), _ptr(sin), cos.shape[0], _ptr(tok_pos), _ptr(err),
             int(halves), _stream()), "rotation of pairs")


def head_gate_(x: torch.Tensor, gate: torch.Tensor, H: int) -> torch.Tensor:
    """In place on x [T, H width] (contiguous): head h of token t times sigmoid(gate[t, h]) (gate a [T, >= H] view)."""
    _need_cuda(x, gate)
    assert x.is_contiguous() and gate.dtype == x.dtype and gate.stride(1) == 1 and x.shape[1] % H == 0
    f = _fn(load_module("latent.cu"), "llb_head_gate", [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _check(f(_ptr(x), _ptr(gate), gate.stride(0), _dt(x), x.shape[0], H, x.shape[1] // H, _stream()), "per-head output gate")
    return x


LATENT_MAX_ROW = 640          # the widest cache row (latent + rotated part) the attention kernel's key tile holds


def require_latent_row(width: int, value_width: int) -> None:
    if not (0 < value_width <= width <= LATENT_MAX_ROW):
        raise KernelError(f"latent attention: cache rows of {width} elements ({value_width} of them the latent) are not supported "
                          f"(at most {LATENT_MAX_ROW})")


def latent_attention(decode: bool, q: torch.Tensor, nh: int, width: int, value_width: int, kv_new: Optional[torch.Tensor],
                     pool: torch.Tensor, page_table: torch.Tensor, ring: int, pinned: int, seq_start: torch.Tensor,
                     seq_len_before: torch.Tensor, n_seqs: int, max_new: int, window: Optional[int], scale: float,
                     sink_logits: Optional[torch.Tensor], n_splits: int = 1) -> torch.Tensor:
    """Softmax attention of nh query heads q [T, nh width] over one shared row per position: the key is the whole row
    [width], the value its first `value_width` elements.  Rows of positions before the step come from the paged pool,
    the step's own from kv_new [T, width] (None: from the pool too, where an earlier call has put them).  Causal, with
    an optional window and a learned sink score per head (float32 [nh]) in the softmax's denominator.
    Returns [T, nh value_width]."""
    _need_cuda(q, kv_new, pool, page_table, sink_logits)
    require_latent_row(width, value_width)
    assert q.dtype == pool.dtype and q.stride(1) == 1 and (kv_new is None or (kv_new.dtype == q.dtype and kv_new.is_contiguous()))
    assert sink_logits is None or (sink_logits.dtype == torch.float32 and sink_logits.numel() == nh)
    out = torch.empty((q.shape[0], nh * value_width), dtype=q.dtype, device=q.device)
    p = _AttnParams()
    p.q, p.row_stride, p.out = q.data_ptr(), q.stride(0), out.data_ptr()
    if kv_new is not None:
        p.k_new, p.kv_row_stride = kv_new.data_ptr(), kv_new.stride(0)
    p.kpool, p.page_table, p.table_stride, p.ring, p.pinned = pool.data_ptr(), page_table.data_ptr(), page_table.shape[1], ring, pinned
    p.seq_start, p.seq_len_before = seq_start.data_ptr(), seq_len_before.data_ptr()
    p.nh, p.nkvh, p.window, p.scale = nh, 1, int(window or 0), scale
    p.all_from_cache = int(kv_new is None)
    p.sink_logits, p.v_in_k, p.n_splits = _ptr(sink_logits), 1, 1
    lib = _attn_lib(width, value_width) if width <= 256 else load_module("attention_simt.cu", {"LLB_HEAD_DIM": width, "LLB_VALUE_DIM": value_width})
    if not decode:
        f = _fn(lib, "llb_attn_prefill", [_AttnParams, c_int, c_int, c_int, c_void_p])
        _check(f(p, _dt(q), n_seqs, max_new, _stream()), "latent attention (prefill)")
        return out
    keep = None
    p.n_splits = n_splits
    if n_splits > 1:
        part_o = torch.empty((n_seqs, nh, n_splits, value_width), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((n_seqs, nh, n_splits, 2), dtype=torch.float32, device=q.device)
        p.part_o, p.part_ml = part_o.data_ptr(), part_ml.data_ptr()
        keep = (part_o, part_ml)
    f = _fn(lib, "llb_attn_decode", [_AttnParams, c_int, c_int, c_void_p])
    _check(f(p, _dt(q), n_seqs, _stream()), "latent attention (decode)", 2 if n_splits > 1 else 1)
    del keep
    return out

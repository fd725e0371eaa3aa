"""Recurrent mechanisms on the GPU: the heads of attention whose values are its keys (csrc/kernels/head_prep.cu), gated linear
attention and time mixing (csrc/kernels/gla.cu), and state-space layers (gla.cu and csrc/kernels/ssd.cu).

Gated linear attention has two kernels.  Portions of at least XFT_GLA_CHUNK_MIN_Q tokens go through the tensor cores in chunks
of 64; shorter ones, decode steps, the 32-bit path and sizes without a chunk instance go token by token.  A batch may hold
both kinds: each kernel takes the sequences whose portions have its length."""
from __future__ import annotations

import ctypes as C

import torch

from . import native as N

NO_LIMIT = (1 << 31) - 1
SMS = 148


def _fn(name):
    f = getattr(N.lib(), name)
    f.restype = C.c_int
    return f


def head_prep(x, d, eps, positions, table, rot, kc, vc, slots, state, state_slots, cu_q, kv_lens, meta=None):
    cu, lens, B, decode, _ = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    assert x.dim() == 2 and x.stride(1) == 1 and kc.dtype == vc.dtype == x.dtype and kc.shape[3] == vc.shape[3] == d.padded
    T, C_ = x.shape[0], (d.hq + d.hkv) * d.dim
    if d.taps > 1:
        assert state.dtype == x.dtype and tuple(state.shape[1:]) == (d.taps - 1, C_) and state.is_contiguous()
    q = torch.empty(T, d.hq, d.padded, dtype=x.dtype, device=x.device)
    ws = N.Workspace.get(x.device)
    nb, _, bs, _ = kc.shape
    rot = rot if table is not None else 0
    N._check(_fn("xft_head_prep")(
        N._p(x), max(x.stride(0), x.shape[1]), T, B, d.hq, d.hkv, d.dim, d.padded, d.taps, N._p(d.conv), N._p(d.q_norm),
        N._p(d.k_norm), C.c_float(eps), N._p(positions), N._p(table), rot, 0 if table is None else table.shape[0], N._p(cu),
        N._p(lens), N._p(state), N._p(state_slots), 0 if state is None else state.shape[0], N._p(q), N._p(kc), N._p(vc), bs,
        C.c_longlong(nb * bs), N._p(slots), int(decode), int(x.dtype == torch.float32), N._p(ws.status), N._stream()),
        f"head_prep (heads of {d.dim}, {d.taps} taps)")
    ws.launches += 1 if decode or d.taps == 1 else 2
    return q


def step_columns(units: int, dim: int, vdim: int) -> int:
    """Columns of a head's state per CTA in the token-by-token kernel: wide enough that a cluster of 8 holds the head, narrow
    enough that `units` (sequence, head) pairs fill the SMs and a thread's share of the state fits its registers."""
    fits = [c for c in (128, 64, 32) if (vdim + c - 1) // c <= 8 and dim <= 32 * 1024 // c]
    if not fits:
        raise N.KernelError(f"gated linear attention: no kernel for states of {dim} x {vdim}")
    best = fits[0]
    for c in fits[1:]:
        if units * ((vdim + best - 1) // best) < 2 * SMS or best >= 2 * vdim or dim * best > 16 * 1024:
            best = c
    return best


def segments(units: int, longest: int) -> int:
    """Segments that run side by side where `units` CTAs alone would leave SMs idle: their two passes over a portion cost about
    one and a half, so it takes more than two of them, of at least four chunks each."""
    n = min(SMS // max(units, 1), longest // (4 * 64), 32)
    return n if n > 1 else 1


def gated_linear(x, d, w, eps, state, state_slots, cu_q, kv_lens, meta=None, out=None):
    cu, lens, B, decode, _ = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    assert x.dim() == 2 and x.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert tuple(state.shape[1:]) == (d.heads, d.dim, d.vdim) and w.a2.dtype == x.dtype and w.a2.is_contiguous()
    T, exact = x.shape[0], x.dtype == torch.float32
    width = d.up(d.heads * d.vdim)                       # the rows of the product that follows
    whole = width == d.heads * d.vdim
    if out is None:
        out = (torch.empty if whole else torch.zeros)(T, width, dtype=x.dtype, device=x.device)
    elif not whole:
        out[:, d.heads * d.vdim:width].zero_()
    ws = N.Workspace.get(x.device)
    f = C.c_float
    common = (N._p(x), max(x.stride(0), x.shape[1]), d.k_at, d.v_at, d.g_at, d.a_at, d.heads, d.dim, d.vdim, d.rank, w.a2.shape[1],
              N._p(w.a2), N._p(w.bias), f(w.tau), f(d.dim ** -0.5 if w.scale is None else w.scale),
              f(eps), N._p(w.bonus), 0 if w.norm.numel() == d.vdim else d.vdim, f(w.mult), N._p(w.norm), N._p(state), N._p(state_slots),
              state.shape[0], N._p(cu), N._p(lens), B)
    columns = 0 if decode or exact else _fn("xft_gla_chunk_columns")(d.dim, d.vdim, d.rank)
    least = NO_LIMIT
    if columns:
        least = max(1, N._ENV().gla_chunk_min_q)
        sizes = [cu_q[i + 1] - cu_q[i] for i in range(B)]
        if max(sizes) >= least:
            raw = torch.empty(T, d.heads * d.vdim, dtype=torch.float32, device=x.device) if d.vdim > columns else None
            long = sum(n >= least for n in sizes)
            segs = segments(long * d.heads * ((d.vdim + columns - 1) // columns), max(sizes))
            ss, sd = (torch.empty(B, d.heads, segs, n, dtype=torch.float32, device=x.device) if segs > 1 else None
                      for n in (d.dim * d.vdim, d.dim))
            N._check(_fn("xft_gla_chunk")(*common, T, N._p(out), out.stride(0), N._p(raw), least, NO_LIMIT, segs, N._p(ss), N._p(sd),
                                          N._p(ws.status), N._stream()), "gla_chunk")
            ws.launches += 1 + (raw is not None) + (segs > 1)
        if min(sizes) >= least:
            return out
    N._check(_fn("xft_gla_step")(*common, N._p(out), out.stride(0), 1, least, step_columns(B * d.heads, d.dim, d.vdim), int(exact),
                                 N._p(ws.status), N._stream()), "gla_step")
    ws.launches += 1
    return out


def token_shift(x, mu, state, state_slots, cu_q, kv_lens, dtype, meta=None):
    cu, lens, B, _, _ = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    n, W = mu.shape
    assert x.dtype == torch.float32 and x.shape[1] == W and x.stride(1) == 1 and tuple(state.shape[1:]) == (W,)
    T = x.shape[0]
    out = torch.empty(T, n * W, dtype=dtype, device=x.device)
    ws = N.Workspace.get(x.device)
    N._check(_fn("xft_token_shift")(N._p(x), max(x.stride(0), W), T, n, W, N._p(mu), N._p(cu), N._p(lens), B, N._p(state), N._p(state_slots),
                                    state.shape[0], N._p(out), int(dtype == torch.float32), N._p(ws.status), N._stream()), "token_shift")
    ws.launches += 1
    return out


def linear_parts(x, W, n, out):
    k, m, T = x.shape[1] // n, W.out_features // n, x.shape[0]
    ldx, ldo = max(x.stride(0), x.shape[1]), max(out.stride(0), out.shape[1])
    ws = N.Workspace.get(x.device)
    assert W.in_features == k and x.dtype == out.dtype and x.stride(1) == out.stride(1) == 1
    if W.kind == "fp32":
        rc = _fn("xft_gemm_f32_heads")(N._p(x), ldx, k, N._p(W.w), N._p(out), ldo, m, n, T, m, k, N._stream())
    elif W.kind != "bf16":
        raise N.KernelError(f"no products side by side for {W.kind} weights")
    elif T > 128:                                        # prompt sizes: the token-major kernel, part by part
        for i in range(n):
            N.gemm_bf16(x[:, i * k:(i + 1) * k], W.w[i * m:(i + 1) * m], m, out=out[:, i * m:(i + 1) * m])
        return out
    else:
        rc = _fn("xft_gemm_bf16_heads")(N._p(x), ldx, x.shape[1], k, N._p(W.w), k, N._p(out), ldo, m, n, T, m, k, N._p(None), 0, 0,
                                        N._p(ws.status), N._stream())
    N._check(rc, "products side by side")
    ws.launches += 1
    return out


def ssd_columns(units: int, state: int, vdim: int) -> int:
    """As `step_columns`, for a kernel whose CTAs of a head need not meet."""
    fits = [c for c in (128, 64, 32) if state <= 32 * 1024 // c]
    if not fits:
        raise N.KernelError(f"state space: no kernel for states of {state} x {vdim}")
    best = fits[0]
    for c in fits[1:]:
        if units * ((vdim + best - 1) // best) < 2 * SMS or best >= 2 * vdim or state * best > 16 * 1024:
            best = c
    return best


def state_space(x, d, w, eps, state, conv_state, state_slots, cu_q, kv_lens, meta=None):
    cu, lens, B, decode, _ = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    assert x.dim() == 2 and x.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert tuple(state.shape[1:]) == (d.heads, d.state, d.vdim)
    assert d.taps == 1 or conv_state.dtype == x.dtype and tuple(conv_state.shape[1:]) == (d.taps - 1, d.channels)
    T, exact, dev = x.shape[0], x.dtype == torch.float32, x.device
    ldx, slots, ns = max(x.stride(0), x.shape[1]), N._p(state_slots), state.shape[0]
    ws = N.Workspace.get(dev)
    f32 = int(exact)
    u = torch.empty(T, d.up(d.channels), dtype=x.dtype, device=dev)
    N._check(_fn("xft_channel_conv")(N._p(x[:, d.x_at:]), ldx, T, B, d.channels, d.taps, N._p(w.conv), N._p(w.conv_bias), N._p(cu), N._p(lens),
                                     N._p(conv_state), slots, ns, N._p(u), u.shape[1], int(decode), f32, N._p(ws.status), N._stream()),
             f"channel_conv ({d.taps} taps)")
    ws.launches += 1 if decode or d.taps == 1 else 2
    y = torch.empty(T, d.inner, dtype=x.dtype, device=dev)
    b_at, c_at, per = d.inner, d.inner + d.groups * d.state, d.heads // d.groups
    dt, vectors = x[:, d.dt_at:], (N._p(w.dt_bias), N._p(w.rate), N._p(w.skip))
    least = NO_LIMIT
    ctas = 0 if decode or exact else _fn("xft_ssd_chunk_ctas")(d.heads, per, d.state, d.vdim)
    if ctas:
        least = max(1, N._ENV().ssd_chunk_min_q)
        sizes = [cu_q[i + 1] - cu_q[i] for i in range(B)]
        if max(sizes) >= least:
            segs = segments(sum(n >= least for n in sizes) * ctas, max(sizes))
            ss, sd = (torch.empty(B, d.heads, segs, n, dtype=torch.float32, device=dev) if segs > 1 else None for n in (d.state * d.vdim, 1))
            N._check(_fn("xft_ssd_chunk")(N._p(u), u.shape[1], b_at, c_at, N._p(dt), ldx, *vectors, d.heads, per, d.state, d.vdim, N._p(state),
                                          slots, ns, N._p(cu), N._p(lens), B, N._p(y), least, segs, N._p(ss), N._p(sd), N._p(ws.status),
                                          N._stream()), "ssd_chunk")
            ws.launches += 1 + (segs > 1)
    if least == NO_LIMIT or min(sizes) < least:
        N._check(_fn("xft_ssd_step")(N._p(u), u.shape[1], c_at, b_at, 0, d.heads, per, d.state, d.vdim, N._p(dt), ldx, *vectors, N._p(state),
                                     slots, ns, N._p(cu), N._p(lens), B, N._p(y), 1, least, ssd_columns(B * d.heads, d.state, d.vdim), f32,
                                     N._p(ws.status), N._stream()), "ssd_step")
        ws.launches += 1
    width = d.up(d.inner)
    out = (torch.empty if width == d.inner else torch.zeros)(T, width, dtype=x.dtype, device=dev)
    N._check(_fn("xft_gated_norm")(N._p(y), d.inner, N._p(x), ldx, N._p(w.norm), N._p(out), width, T, d.norm_groups, d.inner // d.norm_groups,
                                   C.c_float(eps), f32, N._stream()), "gated_norm")
    ws.launches += 1
    return out

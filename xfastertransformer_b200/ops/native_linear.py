"""Recurrent mechanisms on the GPU: the heads of attention whose values are its keys (csrc/kernels/head_prep.cu), and gated
linear attention (csrc/kernels/gla.cu).

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


def gated_linear(x, d, w, eps, state, state_slots, cu_q, kv_lens, meta=None):
    cu, lens, B, decode, _ = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    assert x.dim() == 2 and x.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert tuple(state.shape[1:]) == (d.heads, d.dim, d.vdim) and w.a2.dtype == x.dtype and w.a2.is_contiguous()
    T, exact = x.shape[0], x.dtype == torch.float32
    width = d.up(d.heads * d.vdim)                       # the rows of the product that follows
    out = (torch.empty if width == d.heads * d.vdim else torch.zeros)(T, width, dtype=x.dtype, device=x.device)
    ws = N.Workspace.get(x.device)
    f = C.c_float
    common = (N._p(x), max(x.stride(0), x.shape[1]), d.k_at, d.v_at, d.g_at, d.a_at, d.heads, d.dim, d.vdim, d.rank, w.a2.shape[1],
              N._p(w.a2), N._p(w.bias), f(w.tau), f(d.dim ** -0.5), f(eps), N._p(w.norm), N._p(state), N._p(state_slots),
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

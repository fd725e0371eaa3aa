"""Attention with mixed heads on the GPU: norms and append, and the form for any size (csrc/kernels/talking.cu)."""
from __future__ import annotations

import ctypes as C

import torch

from . import native as N


def _fn(name):
    f = getattr(N.lib(), name)
    f.restype = C.c_int
    return f


def talking_prep(x, d, eps, kc, vc, slots):
    assert x.dim() == 2 and x.stride(1) == 1 and kc.dtype == vc.dtype == x.dtype and kc.shape[3] == vc.shape[3] == d.padded
    T = x.shape[0]
    q = torch.empty(T, d.hq, d.padded, dtype=x.dtype, device=x.device)
    ws = N.Workspace.get(x.device)
    nb, _, bs, _ = kc.shape
    N._check(_fn("xft_talking_prep")(
        N._p(x), max(x.stride(0), x.shape[1]), T, d.k_at, d.hq, d.hkv, d.dim, d.padded, N._p(d.q_norm), N._p(d.k_norm), C.c_float(eps),
        N._p(q), N._p(kc), N._p(vc), bs, C.c_longlong(nb * bs), N._p(slots), int(x.dtype == torch.float32), N._p(ws.status), N._stream()),
        "talking_prep")
    ws.launches += 1
    return q


def talking_attention(q, x, d, kc, vc, block_table, cu_q, kv_lens, scale, window=0, meta=None, out=None):
    cu, lens, B, decode, max_kv = N.batch_arrays(cu_q, kv_lens, meta, q.device)
    T, H, D = q.shape
    assert kc.dtype == q.dtype and x.dtype == q.dtype and q.is_contiguous()
    if out is None:
        out = torch.empty(T, H * D, dtype=q.dtype, device=q.device)
    return _plain(q, x, d, kc, vc, block_table, cu, lens, B, scale, window, out)


def _plain(q, x, d, kc, vc, block_table, cu, lens, B, scale, window, out):
    T, H, D = q.shape
    ws = N.Workspace.get(q.device)
    nb, hkv, bs, _ = kc.shape
    gate = x[:, d.gate_at:]
    f = C.c_float
    N._check(_fn("xft_talking_plain")(
        N._p(q), N._p(gate), max(x.stride(0), x.shape[1]), N._p(out), max(out.stride(0), out.shape[1]), N._p(kc), N._p(vc), N._p(block_table),
        block_table.stride(0), N._p(cu), N._p(lens), B, T, H, hkv, D, bs, nb, f(scale), N._p(d.r1), N._p(d.r2), N._p(d.talk), window,
        f(d.mult), int(q.dtype == torch.float32), N._p(ws.status), N._stream()), f"talking_plain ({H} heads of {D})")
    ws.launches += 1
    return out

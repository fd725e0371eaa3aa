"""Attention with mixed heads on the GPU: norms and append, the form for any size (csrc/kernels/talking.cu), and those for bf16 heads
of 64 or 128 (decode: 256 too) on the tensor cores (csrc/kernels/talking_mma.cu)."""
from __future__ import annotations

import ctypes as C

import torch

from . import native as N

_ENV = N._ENV

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
    if q.dtype == torch.bfloat16 and kc.shape[2] % 64 == 0 and _ENV().talking_tc:
        if decode and can_decode(H, kc.shape[1], D):
            return _decode(q, x, d, kc, vc, block_table, lens, B, max_kv, scale, window, out)
        if kc.shape[2] & (kc.shape[2] - 1) == 0 and _fn("xft_talking_prefill_keys")(H, kc.shape[1], D):
            max_q = meta.max_q if meta is not None and meta.max_q else max(cu_q[i + 1] - cu_q[i] for i in range(B))
            return _prefill(q, x, d, kc, vc, block_table, cu, lens, B, max_q, scale, window, out)
    return _plain(q, x, d, kc, vc, block_table, cu, lens, B, scale, window, out)


def can_decode(hq: int, hkv: int, D: int) -> bool:
    return D in (64, 128, 256) and hq <= 128 and hq // hkv <= 16


def _rows(q, x, d, out):
    """(queries, gate and its stride, output and its stride)"""
    return N._p(q), N._p(x[:, d.gate_at:]), max(x.stride(0), x.shape[1]), N._p(out), max(out.stride(0), out.shape[1])


def decode_splits(units: int, pages: int) -> int:
    """Key ranges of a decode step, a cluster of CTAs: enough for four per SM, at least two pages each."""
    n = 1
    while n < 8 and n * units < 4 * 148 and pages >= 4 * n:
        n *= 2
    return n


def _decode(q, x, d, kc, vc, block_table, lens, B, max_kv, scale, window, out):
    _, H, D = q.shape
    ws = N.Workspace.get(q.device)
    nb, hkv, bs, _ = kc.shape
    pages = (max_kv + 63) // 64
    if window > 0:
        pages = min(pages, (window + 62) // 64 + 1)
    splits = decode_splits(B * hkv, pages)
    f32 = lambda *s: torch.empty(*s, dtype=torch.float32, device=q.device)
    scores, ml = f32(B, H, pages * 64), f32(B, H, splits, 2)
    f = C.c_float
    N._check(_fn("xft_talking_decode")(
        *_rows(q, x, d, out), N._p(kc), N._p(vc), N._p(block_table), block_table.stride(0), N._p(lens), B, H, hkv, D, bs, nb, f(scale),
        N._p(d.r1), N._p(d.r2), N._p(d.talk), window, f(d.mult), splits, pages * 64, N._p(scores), N._p(ml),
        N._p(ws.status), N._stream()), "talking_decode")
    ws.launches += 2
    return out


def _prefill(q, x, d, kc, vc, block_table, cu, lens, B, max_q, scale, window, out):
    _, H, D = q.shape
    ws = N.Workspace.get(q.device)
    nb, hkv, bs, _ = kc.shape
    f = C.c_float
    N._check(_fn("xft_talking_prefill")(
        *_rows(q, x, d, out), N._p(kc), N._p(vc), N._p(block_table), block_table.stride(0), N._p(cu), N._p(lens), B, max_q, H, hkv, D, bs, nb,
        f(scale), N._p(d.r1), N._p(d.r2), N._p(d.talk), window, f(d.mult), N._p(ws.status), N._stream()), "talking_prefill")
    ws.launches += 1
    return out


def _plain(q, x, d, kc, vc, block_table, cu, lens, B, scale, window, out):
    T, H, D = q.shape
    ws = N.Workspace.get(q.device)
    nb, hkv, bs, _ = kc.shape
    f = C.c_float
    N._check(_fn("xft_talking_plain")(
        *_rows(q, x, d, out), N._p(kc), N._p(vc), N._p(block_table),
        block_table.stride(0), N._p(cu), N._p(lens), B, T, H, hkv, D, bs, nb, f(scale), N._p(d.r1), N._p(d.r2), N._p(d.talk), window,
        f(d.mult), int(q.dtype == torch.float32), N._p(ws.status), N._stream()), f"talking_plain ({H} heads of {D})")
    ws.launches += 1
    return out

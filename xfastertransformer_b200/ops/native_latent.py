"""Latent attention of layered designs on the GPU: the step between projection and attention (csrc/kernels/latent.cu), the
per-head products around the cache (gemm_sm100.cu, xft_gemm_bf16_heads) and the attention over latent rows (mla.cu).

Absorbed form (decode and short portions): q' = W_uk^T q per head, so that scores are products of [q' | rotated q] with cache
rows; the weighted sum of latents goes through W_uv per head, and the output gate is the epilogue of that product.  Sizes the
tensor-core kernel does not have, and the 32-bit path, use the plain kernels on the same form.

Expanded form (longer portions): the cache rows that a portion can see are laid next to each other and multiplied with W_uk
and W_uv once, and the portion attends to the result (latent_prefill_sm100.cu).  Per score that is rank / (dim + vdim) of the
absorbed form's work.  A batch may hold both kinds; each sequence takes the form that its own portion asks for."""
from __future__ import annotations

import ctypes as C

import torch

from . import native as N

RANKS = (64, 128, 256, 512)          # latent sizes of the tensor-core kernel
ROT = 64                             # rotated part of its rows


def _fn(name):
    f = getattr(N.lib(), name)
    f.restype = C.c_int
    return f


def latent_prep(x, d, positions, table, rot_dims, norm_w, eps, cache, slots):
    assert x.dim() == 2 and x.stride(1) == 1 and x.dtype in (torch.float32, torch.bfloat16)
    own = d.own_kv
    if own and (cache.dtype != x.dtype or cache.shape[1] != 1 or cache.shape[3] != d.rank + d.rot):
        raise N.KernelError(f"latent cache {tuple(cache.shape)} {cache.dtype} does not fit rows of {d.rank} + {d.rot} in {x.dtype}")
    ws = N.Workspace.get(x.device)
    N._check(_fn("xft_latent_prep")(
        N._p(x), max(x.stride(0), x.shape[1]), x.shape[0], d.heads, d.dim, d.rot, rot_dims if table is not None else 0, d.rank,
        d.rank_real, int(own), N._p(positions), N._p(table), 0 if table is None else table.shape[0], N._p(norm_w if own else None),
        C.c_float(eps), N._p(cache if own else None), C.c_longlong(cache.shape[0] * cache.shape[2]), N._p(slots if own else None),
        int(x.dtype == torch.float32), N._p(ws.status), N._stream()), "latent_prep")
    ws.launches += 1


def _stacked(w, name, make):
    if name not in w.cache:
        w.cache[name] = make().contiguous()
    return w.cache[name]


def _heads(x, ldx, x_cols, xs, w, heads, n_out, k, out, ldo, ys, gate=None, ldg=0, head_gate=False):
    """One product per head (w [heads * n_out, k]) on column ranges of x and out."""
    ws = N.Workspace.get(w.device)
    T = out.shape[0]
    if w.dtype == torch.float32:
        assert gate is None
        rc = _fn("xft_gemm_f32_heads")(N._p(x), ldx, xs, N._p(w), N._p(out), ldo, ys, heads, T, n_out, k, N._stream())
    else:
        rc = _fn("xft_gemm_bf16_heads")(N._p(x), ldx, x_cols, xs, N._p(w), k, N._p(out), ldo, ys, heads, T, n_out, k, N._p(gate), ldg,
                                        int(head_gate), N._p(ws.status), N._stream())
    N._check(rc, "per-head product")
    ws.launches += 1
    return out


EXPAND_BYTES = 2 << 30               # limit of the expanded keys and values of one launch: more heads than fit take turns


def can_expand(d, scale) -> bool:
    """The sizes of attn_flat_tc_kernel: up to 4 chunks of 64 key dimensions, up to 2 of values."""
    return (d.dim % 64 == 0 and d.rot % 64 == 0 and d.vdim % 64 == 0 and d.rot > 0 and d.dim + d.rot <= 256 and d.vdim <= 128
            and d.rank % 8 == 0 and scale > 0)


class _Spans:
    """Which sequences of a batch take the expanded form, and the positions they see."""

    def __init__(self, cu_q, kv_lens, window, least, dev):
        n = range(len(kv_lens))
        ql = [cu_q[i + 1] - cu_q[i] for i in n]
        self.long = [i for i in n if ql[i] >= least]
        self.short = [i for i in n if 0 < ql[i] < least]
        self.max_q = max((ql[i] for i in self.long), default=0)
        lo = [max(0, kv_lens[i] - ql[i] - window + 1) if window > 0 else 0 for i in self.long]
        row, at = [], 0
        for i, a in zip(self.long, lo):
            row.append(at)
            at += kv_lens[i] - a
        self.rows = at
        i32 = lambda x: torch.tensor(x, dtype=torch.int32).to(dev, non_blocking=True)
        if self.long:
            t = i32([self.long, [cu_q[i] for i in self.long], [ql[i] for i in self.long], [kv_lens[i] for i in self.long], lo, row])
            self.seq, self.q_start, self.q_len, self.kv_len, self.lo, self.row = t
        self.part = None
        if self.short and self.long:                 # the short ones become a batch of their own
            cu = [0]
            for i in self.short:
                cu.append(cu[-1] + ql[i])
            seqs, cu_dev, kv = i32(self.short), i32(cu), i32([kv_lens[i] for i in self.short])
            rows = i32([t for i in self.short for t in range(cu_q[i], cu_q[i + 1])])
            self.part = rows, seqs, cu_dev, kv, len(self.short), max(kv_lens[i] for i in self.short)


def latent_attention(x, d, cache, block_table, cu_q, kv_lens, weights, scale, window=0, meta=None, sinks=None):
    cu_dev, kv_dev, B, decode, max_kv = N.batch_arrays(cu_q, kv_lens, meta, x.device)
    out = torch.empty(x.shape[0], d.heads * d.vdim, dtype=x.dtype, device=x.device)
    if decode or x.dtype == torch.float32 or not can_expand(d, scale):
        return _absorbed(x, d, cache, block_table, cu_dev, kv_dev, B, max_kv, weights, scale, window, sinks, out)
    least = N._ENV().latent_expand_min_q
    kept = meta.meta if meta is not None else {}
    key = ("latent spans", window, least)
    sp = kept.get(key)
    if sp is None:
        sp = kept[key] = _Spans(cu_q, kv_lens, window, least, x.device)
    if not sp.long:
        return _absorbed(x, d, cache, block_table, cu_dev, kv_dev, B, max_kv, weights, scale, window, sinks, out)
    _expanded(x, d, cache, block_table, sp, weights, scale, window, sinks, out)
    if sp.part is not None:
        rows, seqs, cu, kv, n, longest = sp.part
        xs = x.index_select(0, rows)
        a = torch.empty(xs.shape[0], d.heads * d.vdim, dtype=x.dtype, device=x.device)
        out.index_copy_(0, rows.long(), _absorbed(xs, d, cache, block_table.index_select(0, seqs), cu, kv, n, longest, weights, scale,
                                                  window, sinks, a))
    return out


def _expanded(x, d, cache, block_table, sp, weights, scale, window, sinks, out):
    """Prompt portions `sp.long` of the rows x into `out`."""
    ws, H, W = N.Workspace.get(x.device), d.heads, d.rank + d.rot
    nb, _, bs, _ = cache.shape
    flat = torch.empty(sp.rows, W, dtype=x.dtype, device=x.device)
    N._check(_fn("xft_latent_gather")(N._p(cache), W, bs, nb, N._p(block_table), block_table.stride(0), N._p(sp.seq), N._p(sp.lo),
                                      N._p(sp.row), len(sp.long), sp.rows, N._p(flat), N._p(ws.status), N._stream()), "latent_gather")
    ws.launches += 1
    per = max(1, min(H, EXPAND_BYTES // (2 * sp.rows * (d.dim + d.vdim))))
    w = _stacked(weights, "ukv", lambda: torch.cat([weights.uk.reshape(H * d.dim, d.rank), weights.uv.reshape(H * d.vdim, d.rank)]))
    for h0 in range(0, H, per):
        n = min(per, H - h0)
        if n == H:
            kv = N.gemm_bf16(flat[:, :d.rank], w, w.shape[0])
        else:
            kv = torch.empty(sp.rows, n * (d.dim + d.vdim), dtype=x.dtype, device=x.device)
            N.gemm_bf16(flat[:, :d.rank], w[h0 * d.dim:(h0 + n) * d.dim], n * d.dim, out=kv[:, :n * d.dim])
            N.gemm_bf16(flat[:, :d.rank], w[H * d.dim + h0 * d.vdim:H * d.dim + (h0 + n) * d.vdim], n * d.vdim, out=kv[:, n * d.dim:])
        flat_attention(x, d, kv, flat, sp, h0, n, scale, window, out, sinks)


def flat_attention(x, d, kv, flat, sp, h0, n, scale, window, out, sinks=None):
    """Heads h0 .. h0 + n - 1 of the packed rows x over expanded keys and values `kv` [rows, n * (dim + vdim)] and the gathered
    cache rows `flat`, which hold the shared key part (csrc/kernels/latent_prefill_sm100.cu)."""
    ws = N.Workspace.get(x.device)
    ldx = max(x.stride(0), x.shape[1])
    gate = x[:, d.gate_at:] if d.gate else None
    N._check(_fn("xft_attn_flat_tc")(
        N._p(x), ldx, d.q_width, d.dim + d.rot, N._p(kv), kv.shape[1], n * d.dim, N._p(flat), flat.shape[1], d.rank, sp.rows,
        N._p(out), out.stride(0), N._p(gate), ldx if d.gate else 0, int(d.head_gate), N._p(sp.q_start), N._p(sp.q_len), N._p(sp.kv_len), N._p(sp.lo),
        N._p(sp.row), len(sp.long), x.shape[0], sp.max_q, h0, n, d.dim // 64, d.rot // 64, d.vdim // 64, C.c_float(scale), N._p(sinks), window,
        N._p(ws.status), N._stream()), "attn_flat_tc")
    ws.launches += 1


# clusters of n CTAs (one CTA per SM) that B200 holds at a time: its GPCs have 16 to 20 SMs
CLUSTERS = {1: 148, 2: 74, 4: 33, 8: 15}


def mla_splits(units: int, keys: int) -> tuple:
    """(CTAs per cluster, clusters) that share the keys of a (token, 16 heads) in the absorbed kernel: as many as run in one
    wave, with at least two 64-key tiles each (eight, where several clusters share them: their merge costs more)."""
    tiles, n, g = (keys + 63) // 64, 1, 1
    while n < 8 and units <= CLUSTERS[2 * n] and tiles >= 4 * n:
        n *= 2
    while g < 8 and 2 * g * units <= CLUSTERS[n] and tiles >= 16 * n * g:
        g *= 2
    return n, g


def mla_scratch(ws, units: int, n: int, g: int, rank: int) -> tuple:
    """(partial outputs, partial maxima and sums, counters) of a launch with `g` clusters per unit."""
    if g == 1:
        return None, None, None
    if units * n > ws.attn_counters.numel():
        raise N.KernelError("latent attention: more partial results than counters")
    return (*ws.attn_partials(units * g * 16 * rank, units * g * n * 32), ws.attn_counters)


def _absorbed(x, d, cache, block_table, cu_dev, kv_dev, B, max_kv, weights, scale, window, sinks, out):
    T, ldx, H, hd = x.shape[0], max(x.stride(0), x.shape[1]), d.heads, d.dim + d.rot
    exact = x.dtype == torch.float32
    wk = _stacked(weights, "uk", lambda: weights.uk.transpose(1, 2).reshape(H * d.rank, d.dim))       # [H * rank, dim]
    wv = _stacked(weights, "uv", lambda: weights.uv.reshape(H * d.vdim, d.rank))
    new = lambda *s: torch.empty(*s, dtype=x.dtype, device=x.device)
    gate = x[:, d.gate_at:] if d.gate else None
    if exact or d.rank not in RANKS or d.rot != ROT:
        q = new(T, H, d.rank + d.rot)
        _heads(x, ldx, d.q_width, hd, wk, H, d.rank, d.dim, q, H * (d.rank + d.rot), d.rank + d.rot)
        q[:, :, d.rank:] = x[:, :d.q_width].view(T, H, hd)[:, :, d.dim:]
        o = N.attention_plain(q, cache, cache, d.rank, block_table, cu_dev, kv_dev, B, scale, H, window=window, sinks=sinks)
        if not exact:
            return _heads(o, H * d.rank, H * d.rank, d.rank, wv, H, d.vdim, d.rank, out, H * d.vdim, d.vdim, gate, ldx, d.head_gate)
        _heads(o, H * d.rank, H * d.rank, d.rank, wv, H, d.vdim, d.rank, out, H * d.vdim, d.vdim)
        if d.gate:
            N._check(_fn("xft_sigmoid_gate")(N._p(out), H * d.vdim, N._p(gate), ldx, N._p(out), H * d.vdim, T, H * d.vdim,
                                             d.vdim if d.head_gate else 1, 1, N._stream()), "sigmoid_gate")
            N.Workspace.get(x.device).launches += 1
        return out
    ws = N.Workspace.get(x.device)
    qa, ol = new(T, H * d.rank), new(T, H * d.rank)
    _heads(x, ldx, d.q_width, hd, wk, H, d.rank, d.dim, qa, H * d.rank, d.rank)
    units = T * ((H + 15) // 16)
    nsplit, groups = mla_splits(units, min(max_kv, window) if window > 0 else max_kv)
    po, pm, cnt = mla_scratch(ws, units, nsplit, groups, d.rank)
    nb, _, bs, _ = cache.shape
    LL = C.c_longlong
    qr = x[:, d.dim:]
    N._check(_fn("xft_mla_attention_ext")(
        N._p(qa), LL(d.rank), LL(H * d.rank), N._p(qr), LL(hd), LL(ldx), N._p(ol), LL(d.rank), LL(H * d.rank), N._p(cache),
        N._p(block_table), block_table.stride(0), N._p(cu_dev), N._p(kv_dev), B, T, H, d.rank, bs, nb, C.c_float(scale), N._p(sinks), window,
        nsplit, groups, N._p(po), N._p(pm), N._p(cnt), N._p(ws.status), N._stream()), "mla_attention")
    ws.launches += 1
    return _heads(ol, H * d.rank, H * d.rank, d.rank, wv, H, d.vdim, d.rank, out, H * d.vdim, d.vdim, gate, ldx, d.head_gate)

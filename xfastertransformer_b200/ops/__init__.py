"""Op entry points.  Device switch only: CPU tensors run `ops.reference` (pure PyTorch),
CUDA tensors run the hand-written sm_100a kernels of `ops.native` (libxft_b200_kernels.so).

There is no silent fallback on a GPU: if the kernel library is missing or an op has no
kernel for the requested variant, the call raises.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from . import reference as R

_native = None


def _nat():
    global _native
    if _native is None:
        import importlib
        _native = importlib.import_module(__name__ + ".native")
    return _native


def _nat_latent():
    from . import native_latent
    return native_latent


def _cuda(t: torch.Tensor) -> bool:
    return t.is_cuda


# -- embedding / norms ----------------------------------------------------------------------
def embedding(ids, table, scale=1.0, out_dtype=torch.float32, pos_table=None, positions=None, pos_offset=0):
    if _cuda(table):
        return _nat().embedding(ids, table, scale, out_dtype, pos_table, positions, pos_offset)
    return R.embedding(ids, table, scale, out_dtype, pos_table, positions, pos_offset)


def rmsnorm(x, w, eps, residual=None):
    if _cuda(x):
        return _nat().rmsnorm(x, w, eps, residual)
    return R.rmsnorm(x, w, eps, residual)


def layernorm(x, w, b, eps):
    if _cuda(x):
        return _nat().layernorm(x, w, b, eps)
    return R.layernorm(x, w, b, eps)


def residual_norm(x, y, post, nxt, eps, kind="layer", rows=None, h_dtype=torch.bfloat16, ids=None, table=None, keep_x=True,
                  embed_scale=1.0, mult=1.0, add=None, raw=False, carry=1.0, post_sum=False):
    """One step of a 32-bit residual stream in one launch: x (or table[ids] * embed_scale) = carry * x + mult * norm(y) with
    `post` = (gain, bias or None) (plain y without it) + the vector `add`, then h = norm(x) with `nxt` for the next product
    (`raw`: x itself).  `post_sum`: `post` normalises the sum instead of y, and its output is the stream.  Returns (x, h); on a GPU x is updated in place unless `rows` selects rows, and buffers are as wide as x (a
    multiple of 8, padding zero)."""
    impl = _nat().residual_norm if _cuda(x if x is not None else table) else R.residual_norm
    return impl(x, y, post, nxt, eps, kind, rows, h_dtype, ids, table, keep_x, embed_scale, mult, add, raw, carry, post_sum)


# -- GEMMs ---------------------------------------------------------------------------------
def _verbose() -> bool:
    from ..utils.flags import Env
    return Env.get().verbose >= 1


def _timed(kernel: str, x, W, fn):
    """XFT_VERBOSE >= 1: run one GEMM-shaped op between two time stamps (device-synchronised on a GPU) and print the
    reference's per-call line ``xft_verbose,exec,<dev>,api,<kernel>,m<M>n<N>k<K>,<ms>`` (src/utils/verbose.h:24-83).
    The decode graph runner steps aside while this is on, so every call is a real launch."""
    import time
    from ..utils import log
    cuda = _cuda(x)
    if cuda:
        torch.cuda.synchronize(x.device)
    t0 = time.perf_counter()
    y = fn()
    if cuda:
        torch.cuda.synchronize(x.device)
    ms = (time.perf_counter() - t0) * 1e3
    log.verbose_line("gpu" if cuda else "cpu", kernel, x.numel() // x.shape[-1], W.out_features, x.shape[-1], ms)
    return y


def linear(x, W, bias=None, act=None, residual=None, res_scale=1.0, out_dtype=None, times=None, out=None):
    """act(x W^T + bias) + res_scale * residual, or with `times` [T, out] act(x W^T + bias) * times.  `out`: rows to write
    into.  act "softcap": res_scale * tanh(. / res_scale)."""
    if out is not None:
        assert residual is None and times is None
        return (_nat() if _cuda(x) else R).linear_into(x, W, bias, act, out)
    if times is not None:
        return (_nat() if _cuda(x) else R).linear_times(x, W, bias, act, times)
    if _verbose():
        name = "gemm" + ("_bias" if bias is not None else "") + (f"_{act}" if act else "") + \
            ("_residual" if residual is not None else "")
        impl = _nat().linear if _cuda(x) else R.linear
        return _timed(name, x, W, lambda: impl(x, W, bias, act, residual, res_scale, out_dtype))
    if _cuda(x):
        return _nat().linear(x, W, bias, act, residual, res_scale, out_dtype)
    return R.linear(x, W, bias, act, residual, res_scale, out_dtype)


def _linear_rms(x, W, eps, bias, act, gated, out_dtype):
    if _cuda(x):
        return _nat().linear_rms(x, W, eps, bias, act, gated, out_dtype)
    h = R.rmsnorm(x, torch.ones(x.shape[-1], dtype=torch.float32), eps)
    return R.linear_gated(h, W, act, bias) if gated else R.linear(h, W, bias, act, None, 1.0, out_dtype)


def linear_rms(x, W, eps, bias=None, act=None, gated=False, out_dtype=None):
    """RMSNorm(x) @ W^T for a weight whose columns already carry the norm's gain (loader.fold_norm_gain)."""
    if _verbose():
        return _timed("rmsnorm_gemm" + ("_gated" if gated else ""), x, W,
                      lambda: _linear_rms(x, W, eps, bias, act, gated, out_dtype))
    return _linear_rms(x, W, eps, bias, act, gated, out_dtype)


def linear_gated(x, W, act="silu", bias=None, limit=0.0):
    """act(g) * u with (g | u) = x W^T + bias; act "clamped": g = min(g, limit), u = u clamped to +-limit, and the result is
    g sigmoid(1.702 g) (u + 1)."""
    impl = _nat().linear_gated if _cuda(x) else R.linear_gated
    if _verbose():
        return _timed(f"gemm_gated_{act}", x, W, lambda: impl(x, W, act, bias, limit))
    return impl(x, W, act, bias, limit)


def linear_parts(x, W, n, out):
    """`n` products side by side: part i of x's columns with rows i of W's n equal parts, into part i of `out`'s columns."""
    impl = _native_linear().linear_parts if _cuda(x) else R.linear_parts
    return impl(x, W, n, out)


def gated_act(gu, act="silu"):
    if _cuda(gu):
        return _nat().gated_act(gu, act)
    return R.gated_act(gu, act)


# -- attention -----------------------------------------------------------------------------
def qkv_rope_cache(qkv, hq, hkv, d, positions, table, rot_dim, style, kc, vc, ks, vs, slots,
                   q_scale=None, q_norm_w=None, k_norm_w=None, eps=1e-6, rot_offset=0, dv=None):
    """Split packed qkv [T,(hq+2hkv)*d] (value heads of size `dv` when given; hkv = 0: query heads only), optional per-head q/k RMSNorm (Qwen3), RoPE on q and k,
    append k/v to the paged cache at `slots` (int8-quantising when scales are given); returns
    q [T,hq,d].  One kernel on the GPU (reference: QKPO + storeKVCache,
    src/layers/attention.h:560-640, src/kernels/attention_kernels.h:45-69)."""
    if _cuda(qkv):
        return _nat().qkv_rope_cache(qkv, hq, hkv, d, positions, table, rot_dim, style, kc, vc, ks, vs, slots,
                                       q_scale, q_norm_w, k_norm_w, eps, rot_offset, dv)
    T = qkv.shape[0]
    q = qkv[:, : hq * d].reshape(T, hq, d)
    k = qkv[:, hq * d:(hq + hkv) * d].reshape(T, hkv, d)
    v = qkv[:, (hq + hkv) * d:].reshape(T, hkv, dv or d)
    if q_norm_w is not None:
        q = R.rmsnorm(q, q_norm_w, eps)
        k = R.rmsnorm(k, k_norm_w, eps)
    if table is not None and rot_dim > 0:
        q, k = R.rope_apply(q, k, positions, table, rot_dim, style, rot_offset, q_scale)
    elif q_scale is not None:
        q = (q.float() * q_scale[:, None, None]).to(q.dtype)
    if hkv > 0:
        R.kv_cache_write(k, v, kc, vc, slots, ks, vs)
    return q.contiguous()


def qkv_rope2d_cache(qkv, hq, hkv, d, positions, positions2, table, kc, vc, ks, vs, slots):
    """ChatGLM-1's two-stream rotary with the cache append: the first half of every q / k head turns by `positions`,
    the second half by `positions2` (block positions), both from one table [max_pos, d/2]; k / v go to the paged cache
    at `slots`; returns q [T,hq,d].  One kernel on the GPU (reference: src/layers/rope_2d.cpp,
    src/models/chatglm.cpp:118-206)."""
    if _cuda(qkv):
        return _nat().qkv_rope2d_cache(qkv, hq, hkv, d, positions, positions2, table, kc, vc, ks, vs, slots)
    T = qkv.shape[0]
    q = qkv[:, : hq * d].reshape(T, hq, d)
    k = qkv[:, hq * d:(hq + hkv) * d].reshape(T, hkv, d)
    v = qkv[:, (hq + hkv) * d:].reshape(T, hkv, d)
    half = d // 2
    q, k = R.rope_apply(q, k, positions, table, half, "half", 0)
    q, k = R.rope_apply(q, k, positions2, table, half, "half", half)
    R.kv_cache_write(k, v, kc, vc, slots, ks, vs)
    return q.contiguous()


def can_fuse_qkv_rope(W, T, D, kc, ks, q_norm_w, k_norm_w, style) -> bool:
    """True when the QKV product, RoPE and the cache append can run as one kernel (GPU, decode sizes)."""
    return _cuda(kc) and _nat().can_fuse_qkv_rope(W, T, D, kc, ks, q_norm_w, k_norm_w, style)


def qkv_linear_rope_cache(x, W, bias, rms_eps, hq, hkv, positions, table, rot_dim, style, kc, vc, slots, q_scale=None):
    """QKV product with split + RoPE + paged cache append as its epilogue; returns q [T, hq, D].  GPU only: callers
    ask can_fuse_qkv_rope first and otherwise run linear / linear_rms followed by qkv_rope_cache."""
    return _nat().qkv_linear_rope_cache(x, W, bias, rms_eps, hq, hkv, positions, table, rot_dim, style, kc, vc, slots,
                                        q_scale)


def paged_attention(q, kc, vc, block_table, cu_q, kv_lens, scale, ks=None, vs=None, slopes=None,
                    causal=True, prefix_lm_lens=None, group=None, q_off=0, meta=None, softcap=0.0, window=0, keep_first=0,
                    sinks=None):
    """Attention of a ragged batch over the paged cache; `softcap`, `window` with `keep_first`, and `sinks` as in
    `reference.paged_attention`."""
    if _cuda(q):
        return _nat().paged_attention(q, kc, vc, block_table, cu_q, kv_lens, scale, ks, vs, slopes,
                                        causal, prefix_lm_lens, group, q_off, meta, softcap, window, keep_first, sinks)
    return R.paged_attention(q, kc, vc, block_table, cu_q, kv_lens, scale, ks, vs, slopes, causal,
                             prefix_lm_lens, group, q_off, softcap, window, keep_first, sinks)


def mla_attention(q_nope, q_rope, latent_cache, block_table, cu_q, kv_lens, w_uk, w_uv, scale, absorbed=True,
                  meta=None):
    if _cuda(q_nope):
        return _nat().mla_attention(q_nope, q_rope, latent_cache, block_table, cu_q, kv_lens, w_uk, w_uv,
                                      scale, absorbed, meta)
    return R.mla_attention(q_nope, q_rope, latent_cache, block_table, cu_q, kv_lens, w_uk, w_uv, scale, absorbed)


def rope_apply(q, k, positions, table, rot_dim, style="half", rot_offset=0, q_scale=None):
    if _cuda(q):
        return _nat().rope_apply(q, k, positions, table, rot_dim, style, rot_offset, q_scale)
    return R.rope_apply(q, k, positions, table, rot_dim, style, rot_offset, q_scale)


def latent_cache_write(latent, cache, slots):
    """latent [T, kv_lora+rope] -> cache [nb,1,block,kv_lora+rope] at `slots`."""
    if _cuda(latent):
        return _nat().latent_cache_write(latent, cache, slots)
    blk = cache.shape[2]
    cache[(slots // blk).long(), 0, (slots % blk).long()] = latent.to(cache.dtype)


def mla_prep(q, kv, Hl, nope, rope, kvl, positions, table, kv_norm_w, eps, cache, slots):
    """What sits between the MLA projections and the MLA attention: split every query head of q [T, Hl*(nope+rope)]
    into its no-position part and its rotated part (interleaved pairs), RMS-normalise the compressed KV kv[:, :kvl],
    rotate the shared key part kv[:, kvl:], and append (normalised KV ‖ rotated key) to the latent cache at `slots`.
    Returns (q_nope [T,Hl,nope], q_rope [T,Hl,rope]).  One kernel on the GPU."""
    if _cuda(q) and cache.dtype == torch.bfloat16:
        return _nat().mla_prep(q, kv, Hl, nope, rope, kvl, positions, table, kv_norm_w, eps, cache, slots)
    T = q.shape[0]
    q3 = q.reshape(T, Hl, nope + rope)
    ckv = R.rmsnorm(kv[:, :kvl], kv_norm_w, eps)
    q_rope, kr = R.rope_apply(q3[..., nope:], kv[:, kvl:].reshape(T, 1, rope), positions, table, rope, "interleaved", 0)
    latent_cache_write(torch.cat([ckv, kr.reshape(T, rope)], dim=-1), cache, slots)
    return q3[..., :nope].contiguous(), q_rope.contiguous()


@dataclass(frozen=True)
class LatentDims:
    """Sizes of a latent-attention layer as its kernels see them (heads of this rank; sizes possibly padded with zeros).
    A packed row is [q: heads x (dim + rot) | latent: rank + rot (unless the layer reads another's) | gate: heads x vdim], or
    with `head_gate` one gate value per head, in a row of a multiple of `align` values."""
    heads: int
    dim: int                    # unrotated query/key dimensions per head
    rot: int                    # rotated dimensions per head
    rank: int                   # latent
    vdim: int
    own_kv: bool
    gate: bool
    rank_real: int              # values of the latent that are not padding (the norm's count)
    head_gate: bool = False
    align: int = 1

    @property
    def q_width(self) -> int:
        return self.heads * (self.dim + self.rot)

    @property
    def gate_at(self) -> int:
        return self.q_width + (self.rank + self.rot if self.own_kv else 0)

    @property
    def row(self) -> int:
        n = self.gate_at + (0 if not self.gate else self.heads if self.head_gate else self.heads * self.vdim)
        return (n + self.align - 1) // self.align * self.align


def latent_prep(x, dims: LatentDims, positions, table, rot_dims, norm_w, eps, cache, slots):
    """What sits between the packed projection x [T, dims.row] of a latent-attention layer and its attention: rotates the
    rotated part of every query in place (interleaved pairs, the first `rot_dims`), and, for a layer with a cache of its
    own, appends [RMS-normed latent | rotated key part] to `cache` [blocks, 1, block, rank + rot] at `slots`."""
    if _cuda(x):
        return _nat_latent().latent_prep(x, dims, positions, table, rot_dims, norm_w, eps, cache, slots)
    d, T = dims, x.shape[0]
    q = x[:, :d.q_width].view(T, d.heads, d.dim + d.rot)
    kr = x[:, d.q_width + d.rank:d.q_width + d.rank + d.rot].reshape(T, 1, d.rot) if d.own_kv else None
    if table is not None and rot_dims > 0:
        qr, kr = R.rope_apply(q[..., d.dim:], kr, positions, table, rot_dims, "interleaved")
        q[..., d.dim:] = qr
    if d.own_kv:
        c = x[:, d.q_width:d.q_width + d.rank].float()
        n = c * torch.rsqrt(c.pow(2).sum(-1, keepdim=True) / d.rank_real + eps) * norm_w
        latent_cache_write(torch.cat([n.to(x.dtype), kr.reshape(T, d.rot)], -1), cache, slots)


def latent_attention(x, dims: LatentDims, cache, block_table, cu_q, kv_lens, weights, scale, window=0, meta=None, sinks=None):
    """Attention of the packed rows x (after `latent_prep`) over a latent cache -> [T, heads * vdim], multiplied with the
    sigmoid of the rows' gate.  `weights`: `LatentWeights`.  `window` and `sinks` as in `paged_attention`."""
    if _cuda(x):
        return _nat_latent().latent_attention(x, dims, cache, block_table, cu_q, kv_lens, weights, scale, window, meta, sinks)
    d, T = dims, x.shape[0]
    q = x[:, :d.q_width].view(T, d.heads, d.dim + d.rot)
    a = R.mla_attention(q[..., :d.dim], q[..., d.dim:], cache, block_table, cu_q, kv_lens, weights.uk, weights.uv, scale,
                        max(cu_q[i + 1] - cu_q[i] for i in range(len(kv_lens))) == 1, window, sinks).reshape(T, -1)
    if d.gate and d.head_gate:
        g = torch.sigmoid(x[:, d.gate_at:d.gate_at + d.heads].float())[:, :, None]
        a = (a.view(T, d.heads, d.vdim).float() * g).to(a.dtype).reshape(T, -1)
    elif d.gate:
        a = (a.float() * torch.sigmoid(x[:, d.gate_at:d.gate_at + d.heads * d.vdim].float())).to(a.dtype)
    return a


class LatentWeights:
    """The per-head matrices of a latent-attention layer: uk [heads, dim, rank], uv [heads, vdim, rank]."""

    def __init__(self, uk, uv):
        self.uk, self.uv = uk.contiguous(), uv.contiguous()
        self.cache: dict = {}               # layouts the kernels want, made once


# -- attention whose values are its keys ------------------------------------------------------
@dataclass
class HeadPrep:
    """What happens to the heads of a packed row [q: hq x dim | k: hkv x dim] between projection and cache: weights of the
    short convolution [taps, (hq + hkv) * dim] fp32 (None: none), gains of the norms per head (None: none).  Heads leave
    `padded` wide, zeros behind `dim`."""
    hq: int
    hkv: int
    dim: int
    padded: int
    conv: Optional[torch.Tensor]
    q_norm: Optional[torch.Tensor]
    k_norm: Optional[torch.Tensor]

    @property
    def taps(self) -> int:
        return 1 if self.conv is None else self.conv.shape[0]


def head_prep(x, prep: HeadPrep, eps, positions, table, rot_dims, kc, vc, slots, state, state_slots, cu_q, kv_lens, meta=None):
    """Causal convolution over time on every channel of q and k, RMS norm per head, rotation of the first `rot_dims`
    dimensions; appends k to `kc` and the keys as they left the convolution to `vc`, and returns q [T, hq, padded].
    `state` [slots, taps - 1, channels] holds the last inputs of each sequence's convolution, oldest first, and is moved on
    to the end of this call's tokens; what lies before a sequence's first token counts as zero."""
    impl = _native_linear().head_prep if _cuda(x) else R.head_prep
    return impl(x, prep, eps, positions, table, rot_dims, kc, vc, slots, state, state_slots, cu_q, kv_lens, meta)


# -- gated linear attention -------------------------------------------------------------------
@dataclass(frozen=True)
class LinearDims:
    """A packed row of a gated-linear-attention layer: [q: heads x dim | k | v: heads x vdim | g | a1: rank], each part
    starting at a multiple of `align` values."""
    heads: int
    dim: int
    vdim: int
    rank: int
    align: int = 1

    def up(self, n: int) -> int:
        return (n + self.align - 1) // self.align * self.align

    @property
    def k_at(self) -> int:
        return self.up(self.heads * self.dim)

    @property
    def v_at(self) -> int:
        return 2 * self.k_at

    @property
    def g_at(self) -> int:
        return self.v_at + self.up(self.heads * self.vdim)

    @property
    def a_at(self) -> int:
        return self.g_at + self.up(self.heads * self.vdim)


@dataclass
class LinearWeights:
    """Decay and output norm: the decay's second product a2 [heads * dim, rank (aligned)] and its bias, `tau`, the gain of
    the norm over a head's vdim outputs ([vdim], or [heads * vdim]).  `scale` of the queries (None: 1 / sqrt(dim)).  `bonus`
    [heads, dim]: the current token is read with this factor on its key instead of through the state, and decays are
    exp(-exp(z)).  `mult`: a factor of the result."""
    a2: torch.Tensor
    bias: torch.Tensor
    tau: float
    norm: torch.Tensor
    scale: Optional[float] = None
    bonus: Optional[torch.Tensor] = None
    mult: float = 1.0


def gated_linear(x, dims: LinearDims, w: LinearWeights, eps, state, state_slots, cu_q, kv_lens, meta=None, out=None):
    """Gated linear attention of packed rows x -> [T, heads * vdim (aligned)] (into `out` when given).  Per head, with z = W_a2 a1
    + bias and decay = sigmoid(z)^(1 / tau) per key channel: S <- diag(decay) S + k v^T and o = S^T (q * scale); the result is
    norm(o) * silu(g).  With a bonus u: decay = exp(-exp(z)), and o = (S + diag(u) k v^T)^T q is read before S moves on.
    `state` [slots, heads, dim, vdim] fp32 is carried on; a sequence's first token starts from zero."""
    impl = _native_linear().gated_linear if _cuda(x) else R.gated_linear
    return impl(x, dims, w, eps, state, state_slots, cu_q, kv_lens, meta, out)


def token_shift(x, mu, state, state_slots, cu_q, kv_lens, dtype, meta=None):
    """Mixes of every row with the row of the token before it: column part i of the result [T, n * width] is
    x + (previous x - x) * mu[i] (mu [n, width] fp32), the arithmetic in fp32.  `state` [slots, width] fp32 holds the last row of
    each sequence and is moved on; in front of a sequence's first token are zeros."""
    impl = _native_linear().token_shift if _cuda(x) else R.token_shift
    return impl(x, mu, state, state_slots, cu_q, kv_lens, dtype, meta)


# -- state-space recurrence ---------------------------------------------------------------------
@dataclass(frozen=True)
class StateDims:
    """A packed row of a state-space layer: [z: heads x vdim | x: heads x vdim, B, C: groups x state each | dt: heads]; the three
    parts start at multiples of `align` values, and x, B, C are one run of channels."""
    heads: int
    state: int
    vdim: int
    groups: int
    norm_groups: int
    taps: int
    align: int = 1

    def up(self, n: int) -> int:
        return (n + self.align - 1) // self.align * self.align

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def x_at(self) -> int:
        return self.up(self.inner)

    @property
    def dt_at(self) -> int:
        return self.x_at + self.up(self.channels)

    @property
    def row(self) -> int:
        return self.dt_at + self.up(self.heads)


@dataclass
class StateWeights:
    """fp32: the convolution [taps, channels] and its bias, per head dt_bias, the decay's rate exp(A_log) and the skip's factor D,
    the gain of the output norm [heads * vdim]."""
    conv: torch.Tensor
    conv_bias: torch.Tensor
    dt_bias: torch.Tensor
    rate: torch.Tensor
    skip: torch.Tensor
    norm: torch.Tensor


def state_space(x, dims: StateDims, w: StateWeights, eps, state, conv_state, state_slots, cu_q, kv_lens, meta=None):
    """The mixer of a state-space layer between its two projections, packed rows x -> [T, heads * vdim (aligned)]: x, B and C
    through a causal convolution and silu, dt through softplus, then per head S <- exp(-rate dt) S + dt B x^T and
    y = S^T C + D x; y * silu(z) is normalised in `norm_groups` parts.  `state` [slots, heads, state, vdim] fp32 and `conv_state`
    [slots, taps - 1, channels] (None for one tap) are carried on; a sequence's first token starts from zero."""
    impl = _native_linear().state_space if _cuda(x) else R.state_space
    return impl(x, dims, w, eps, state, conv_state, state_slots, cu_q, kv_lens, meta)


# -- attention with mixed heads -----------------------------------------------------------------
@dataclass
class TalkingHeads:
    """Attention whose heads' weights are mixed.  A packed row is [q: hq x dim | k: hkv x dim | gate: hq x padded], each part starting
    at a multiple of `align` values; heads leave `padded` wide.  Gains of the norms over the whole projections [hq * dim] and
    [hkv * dim], the distance bias r1, r2 [hq], the mixing matrix talk [hq, hq], all fp32.  `mult`: a factor of the result."""
    hq: int
    hkv: int
    dim: int
    padded: int
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    r1: torch.Tensor
    r2: torch.Tensor
    talk: torch.Tensor
    mult: float = 1.0
    align: int = 1

    def up(self, n: int) -> int:
        return (n + self.align - 1) // self.align * self.align

    @property
    def k_at(self) -> int:
        return self.up(self.hq * self.dim)

    @property
    def gate_at(self) -> int:
        return self.k_at + self.up(self.hkv * self.dim)

    @property
    def row(self) -> int:
        return self.gate_at + self.up(self.hq * self.padded)


def talking_prep(x, d: TalkingHeads, eps, kc, vc, slots):
    """RMS norms over all of a row's q and over all of its k; appends k to `kc` and k as it was before its norm to `vc`, and
    returns q [T, hq, padded]."""
    return (_native_talking() if _cuda(x) else R).talking_prep(x, d, eps, kc, vc, slots)


def talking_attention(q, x, d: TalkingHeads, kc, vc, block_table, cu_q, kv_lens, scale, window=0, meta=None, out=None):
    """Attention with scores q . k * scale - r1 ln(1 + r2 (i - j)) over the keys that `window` leaves, a softmax per head, the heads'
    weights mixed by `talk` (head h applies sum_g talk[h, g] weight_g to the values of its own key/value head), and the gate of
    the packed rows x: -> [T, hq * padded] (into `out` when given)."""
    impl = (_native_talking() if _cuda(q) else R).talking_attention
    return impl(q, x, d, kc, vc, block_table, cu_q, kv_lens, scale, window, meta, out)


def _native_talking():
    from . import native_talking
    return native_talking


def _native_linear():
    from . import native_linear
    return native_linear


# -- MoE -----------------------------------------------------------------------------------
def route(logits, kind, top_k, bias=None, n_group=1, topk_group=1, routed_scaling=1.0, norm_topk=True,
          scoring="sigmoid"):
    if _cuda(logits):
        return _nat().route(logits, kind, top_k, bias, n_group, topk_group, routed_scaling, norm_topk, scoring)
    if kind == "mixtral":
        return R.route_mixtral(logits, top_k)
    if kind == "softmax_topk":
        return R.route_softmax_topk(logits, top_k, norm_topk)
    if kind == "deepseek":
        return R.route_deepseek(logits, bias, top_k, n_group, topk_group, routed_scaling, norm_topk, scoring)
    raise ValueError(kind)


def moe_experts(x, idx, w, experts, act="silu", expert_offset=0, packed=None, expected_pairs=None, gated=True, add=None):
    """Weighted sum of the chosen experts' outputs (see `reference.moe_experts`) in fp32, plus `add` [T, H] fp32."""
    if _cuda(x):
        return _nat().moe_experts(x, idx, w, experts, act, expert_offset, packed, expected_pairs, gated, add)
    out = R.moe_experts(x, idx, w, experts, act, expert_offset, gated)
    return out if add is None else out + add


# -- sampling ------------------------------------------------------------------------------
def argmax_rows(logits):
    if _cuda(logits):
        return _nat().argmax_rows(logits)
    return R.argmax_rows(logits)


def beam_topk(logits, k):
    """(log-softmax values, token ids) of each row's k best entries, best first."""
    if _cuda(logits):
        from . import native_sample
        return native_sample.beam_topk(logits, k)
    return R.beam_topk(logits, k)


def sample_top_k_top_p(logits, top_k, top_p, temperature, uniform):
    if _cuda(logits):
        return _nat().sample_top_k_top_p(logits, top_k, top_p, temperature, uniform)
    return R.sample_top_k_top_p(logits, top_k, top_p, temperature, uniform)

"""Layered designs (Kafipel, Vepivik, Botusun, Dagezen) on a GPU: every kernel of the path alone, and whole models in bf16 and in 32 bits, against a
plain implementation of the equations."""
import os
import sys

import pytest
import torch

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "tests"))

import layered_cases as C  # noqa: E402
import layered_ops_cases as M  # noqa: E402
import oracle_layered as O  # noqa: E402
import xfastertransformer_b200 as xft  # noqa: E402

BF16_TOL = 1.2e-2                # a product of bf16 operands against fp64 on the same operands


def _dev():
    return torch.device("cuda", 0)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    root, made = tmp_path_factory.mktemp("layered"), {}

    def get(name):
        if name not in made:
            made[name] = C.Case(root, name)
        return made[name]
    return get


# ------------------------------------------------------------------------------------------ attention kernels
@pytest.mark.parametrize("window,keep", [(40, 5), (64, 64), (1, 3), (129, 2), (33, 70)])
@pytest.mark.parametrize("d,decode", [(64, False), (64, True), (128, False), (128, True), (256, False), (256, True)])
def test_window_edges_bf16(d, decode, window, keep):
    """mma.sync prompt kernels (64, 256), the tcgen05 prompt kernel (128), the TMA-ring decode kernel."""
    M.window_edges(_dev(), torch.bfloat16, d, d, window, keep, decode, BF16_TOL)


@pytest.mark.parametrize("window,keep", [(40, 5), (129, 2), (1, 0)])
@pytest.mark.parametrize("d", [64, 128])
def test_window_edges_cp_async_decode(d, window, keep, monkeypatch):
    from xfastertransformer_b200.utils.flags import Env
    monkeypatch.setenv("XFT_ATTN_TMA", "0")
    Env.get().reload()
    M.window_edges(_dev(), torch.bfloat16, d, d, window, keep, True, BF16_TOL)


@pytest.mark.parametrize("splits", [2, 5])
def test_window_edges_split_decode(splits, monkeypatch):
    """Several CTAs per (sequence, head): the sink counts in one of them, the kept tiles may be another's."""
    from xfastertransformer_b200.utils.flags import Env
    monkeypatch.setenv("XFT_ATTN_SPLITS", str(splits))
    Env.get().reload()
    M.window_edges(_dev(), torch.bfloat16, 128, 128, 129, 2, True, BF16_TOL)
    M.sink_counts_once(_dev(), torch.bfloat16, 128, BF16_TOL, T=330)


def test_tc_prompt_kernel_off(monkeypatch):
    from xfastertransformer_b200.utils.flags import Env
    monkeypatch.setenv("XFT_ATTN_TC_MIN_Q", "1000000")
    Env.get().reload()
    M.window_edges(_dev(), torch.bfloat16, 128, 128, 40, 5, False, BF16_TOL)


@pytest.mark.parametrize("window,keep", [(40, 5), (64, 64), (1, 0), (129, 2)])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)])
def test_window_edges_plain_kernel(dtype, tol, decode, window, keep):
    M.window_edges(_dev(), dtype, 40, 24, window, keep, decode, tol)


@pytest.mark.parametrize("d", [64, 128, 256])
def test_sinks_and_cap_bf16(d):
    M.sink_counts_once(_dev(), torch.bfloat16, d, BF16_TOL)
    M.softcap(_dev(), torch.bfloat16, d, BF16_TOL)


def test_sinks_and_cap_fp32():
    M.sink_counts_once(_dev(), torch.float32, 36, 3e-6)
    M.softcap(_dev(), torch.float32, 36, 3e-6)


@pytest.mark.parametrize("d,pad", [(20, 64), (80, 128), (136, 256)])
def test_padded_heads(d, pad):
    for decode in (False, True):
        M.window_edges(_dev(), torch.bfloat16, d, d - 4, 40, 5, decode, BF16_TOL, pad=pad)


@pytest.mark.parametrize("group", [1, 6, 20])
def test_group_sizes(group):
    """More query heads per key/value head than one CTA's 16 rows."""
    for decode in (False, True):
        M.window_edges(_dev(), torch.bfloat16, 128, 128, 70, 3, decode, BF16_TOL, H=group * 2, G=2)


def test_far_keys_among_many():
    """One key thousands of positions back, inside a wide window or kept, found by prompt portions and decode steps."""
    T = 2100
    for window, keep, j in ((1900, 2, 250), (64, 130, 129), (64, 130, 130), (2000, 0, 99), (2000, 0, 101)):
        q, k, v = M._inputs(T, 2, 1, 128, 128, torch.bfloat16, j)
        q[..., 0], k[..., 0] = 3.0, 0.0
        k[j, :, 0] = 8.0
        sink = torch.tensor([0.5, -2.0])
        want = O.attention(q.double(), k.double(), v.double(), 1.0, 50.0, {"size": window, "keep_first": keep}, sink.double())
        for decode in (False, True):
            got = M.attend(_dev(), torch.bfloat16, q, k, v, decode, T - 60, scale=1.0, softcap=50.0, window=window,
                           keep_first=keep, sinks=sink.cuda())
            M._close(got, want[T - 60:].float(), BF16_TOL, f"window {window}, kept {keep}, key {j}, decode {decode}")


# ------------------------------------------------------------------------------------------ other kernels
@pytest.mark.parametrize("H", [72, 100, 256, 1021, 1536, 3000, 5120, 12288, 20000])
@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_residual_norm(H, kind):
    M.residual_norm(_dev(), H, kind, torch.bfloat16, torch.bfloat16, 4e-6)
    M.residual_norm(_dev(), H, kind, torch.float32, torch.float32, 4e-6)


@pytest.mark.parametrize("T,N,K", [(1, 130, 77), (65, 64, 16), (200, 333, 1000)])
def test_gemm_f32(T, N, K):
    """True 32-bit products: a reduced-precision mode would be off by 1e-3."""
    from xfastertransformer_b200.ops import native as N_
    from xfastertransformer_b200.runtime.loader import make_linear
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(T, K, generator=g), torch.randn(2 * N, K, generator=g)
    want = x.double() @ w.double().T
    W = make_linear(w.cuda(), "fp32")
    got = N_.linear(x.cuda(), W)
    assert float((got.double().cpu() - want).abs().max() / want.abs().max()) < 2e-6
    gate, up = want[:, :N], want[:, N:]
    got = N_.linear_gated(x.cuda(), W, "silu")
    ref = gate * torch.sigmoid(gate) * up
    assert float((got.double().cpu() - ref).abs().max() / ref.abs().max()) < 2e-6


@pytest.mark.parametrize("dtype,d,dv,tol", [(torch.float32, 40, 24, 2e-5), (torch.bfloat16, 264, 272, 8e-3), (torch.bfloat16, 64, 64, 8e-3)])
def test_rotation(dtype, d, dv, tol):
    M.rotation(_dev(), dtype, {"dims": 24, "base": 900.0, "scaling": {"factor": 3.0, "original": 50, "fast": 5.0, "slow": 0.5}},
               d, dv, tol)


# ------------------------------------------------------------------------------------------ latent attention, experts
FORMS = pytest.mark.parametrize("form", ["decode", "portion", "short portion", "mixed"])


def _form(monkeypatch, form):
    """(decode steps?, extra short portions) of a form; "short portion" keeps a long portion in the absorbed form."""
    from xfastertransformer_b200.utils.flags import Env
    monkeypatch.setenv("XFT_LATENT_EXPAND_MIN_Q", "100000" if form == "short portion" else "16")
    Env.get().reload()
    return form == "decode", 2 if form == "mixed" else 0


@FORMS
@pytest.mark.parametrize("window", [40, 64, 1, 129, 0])
def test_latent_window_edges(monkeypatch, form, window):
    decode, extra = _form(monkeypatch, form)
    M.latent_window_edges(_dev(), torch.bfloat16, window, decode, BF16_TOL, extra=extra)
    M.latent_window_edges(_dev(), torch.bfloat16, window, decode, BF16_TOL, H=17, d=128, rd=64, R=200, dv=128, extra=extra)


@FORMS
@pytest.mark.parametrize("sizes", [dict(H=2, d=208, rd=80, R=520, dv=144), dict(H=3, d=136, rd=24, R=300, dv=72),
                                   dict(H=33, d=64, rd=64, R=512, dv=64), dict(H=4, d=16, rd=2, R=12, dv=8)])
def test_latent_sizes(monkeypatch, form, sizes):
    """Sizes without a tensor-core kernel, three key chunks, more than 16 heads per token twice over, very small ones."""
    decode, extra = _form(monkeypatch, form)
    M.latent_window_edges(_dev(), torch.bfloat16, 70, decode, BF16_TOL, extra=extra, **sizes)
    M.latent_heads_differ(_dev(), torch.bfloat16, BF16_TOL, decode, extra=extra, **sizes)


@pytest.mark.parametrize("window", [40, 129, 0])
@pytest.mark.parametrize("decode", [False, True])
def test_latent_fp32(window, decode):
    M.latent_window_edges(_dev(), torch.float32, window, decode, 5e-6)
    M.latent_heads_differ(_dev(), torch.float32, 5e-6, decode)


def test_latent_far_keys(monkeypatch):
    """A key thousands of positions back, just inside and just outside a wide window, in split decode steps and in portions
    of several key tiles whose maxima grow from tile to tile."""
    T = 2100
    q, c, kr, uk, uv, gate = M._latent_layer(2, 64, 32, 100, 64, T, 1)
    q[..., 64], kr[:, 0] = 3.0, 0.0
    kr[:, 1], q[..., 65] = torch.arange(T) / 300.0, 2.0            # later keys weigh more: the running maximum rises
    for window, j in ((1900, 250), (1900, 180), (2000, 99), (2000, 101), (0, 5)):
        k2 = kr.clone()
        k2[j, 0] = 12.0
        want = M.latent_want(q, c, k2, uk, uv, gate, 1.0, window)
        for form in ("decode", "portion", "short portion"):
            decode, _ = _form(monkeypatch, form)
            for start in (T - 60,) if form != "portion" else (T - 60, T - 700):
                got = M.latent_run(_dev(), torch.bfloat16, q, c, k2, uk, uv, gate, 1.0, window, decode, start)
                M._close(got, want[start:], BF16_TOL, f"window {window}, key {j}, {form}")


def test_latent_expanded_by_head_groups(monkeypatch):
    from xfastertransformer_b200.ops import native_latent
    monkeypatch.setattr(native_latent, "EXPAND_BYTES", 7 * 2 * 150 * (64 + 64))
    M.latent_heads_differ(_dev(), torch.bfloat16, BF16_TOL, False, window=0)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
def test_latent_prep(dtype, tol):
    M.latent_prep(_dev(), dtype, tol)
    M.latent_prep(_dev(), dtype, tol, T=3, H=33, d=64, rd=64, R=512, spare=0)


@pytest.mark.parametrize("T,E,top,ff,shared", [(9, 5, 2, 24, 40), (1, 7, 7, 8, 0), (300, 33, 3, 64, 128), (200, 1, 1, 136, 8)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_experts(dtype, tol, T, E, top, ff, shared):
    M.experts(_dev(), dtype, tol, T, E, top, ff, shared)


# ------------------------------------------------------------------------------------------ recurrent mechanisms
KINDS = pytest.mark.parametrize("dtype,tol", [(torch.float32, 4e-5), (torch.bfloat16, 1.5e-2)])


@KINDS
@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 40, 3, 17), (64, 200, 16, 65)])
@pytest.mark.parametrize("H,d,dv,rank,tau", [(3, 12, 20, 5, 4.0), (2, 128, 128, 16, 16.0), (2, 40, 64, 33, 1.0), (2, 72, 80, 24, 9.0)])
def test_gated_linear(dtype, tol, H, d, dv, rank, tau, sizes):
    """Token by token, in chunks, and both in one batch."""
    n = 70 if max(sizes) < 3 else 300
    M.gated_linear(_dev(), dtype, tol, H, d, dv, rank, tau, (n, 33, 1, 130, 6), sizes)


@KINDS
@pytest.mark.parametrize("H,d,dv,rank", [(1, 200, 144, 16), (2, 256, 64, 9), (1, 300, 72, 9), (2, 33, 21, 7), (1, 8, 8, 1), (1, 64, 520, 64),
                                         (5, 128, 192, 48), (1, 512, 256, 16)])
def test_gated_linear_sizes(dtype, tol, H, d, dv, rank):
    """Columns over several CTAs, sizes without a chunk instance, odd sizes, clusters of many."""
    M.gated_linear(_dev(), dtype, tol, H, d, dv, rank, 12.0, (100, 20, 3), (1000,))
    M.gated_linear(_dev(), dtype, tol, H, d, dv, rank, 12.0, (20, 3), (1, 2))


@KINDS
@pytest.mark.parametrize("tau,around,spread", [(0.2, 0.0, 3.0), (1.0, -3.0, 2.0), (0.05, 1.0, 2.0), (2.0, -9.0, 6.0), (16.0, 5.0, 0.5)])
def test_gated_linear_decays(dtype, tol, tau, around, spread):
    """Decays from none to all within a token: chunks in one piece, in pieces, and pieces from differences."""
    M.gated_linear(_dev(), dtype, tol, 2, 64, 64, 16, tau, (200, 65, 17), (1000,), around, spread)
    M.gated_linear(_dev(), dtype, tol, 1, 136, 40, 16, tau, (90,), (1000,), around, spread)


@pytest.mark.parametrize("H,d,dv,tau", [(2, 64, 64, 16.0), (1, 128, 128, 4.0), (1, 136, 100, 16.0), (2, 24, 40, 0.5)])
@pytest.mark.parametrize("sizes", [(2000,), (900, 1400)])
def test_gated_linear_segments(H, d, dv, tau, sizes):
    """Few long portions go in segments that run side by side, beside portions of one chunk and of one token."""
    M.gated_linear(_dev(), torch.bfloat16, 1.5e-2, H, d, dv, 16, tau, (1500, 70, 1130, 33, 3), sizes)


@pytest.mark.parametrize("columns", [32, 64, 128])
def test_gated_linear_step_columns(monkeypatch, columns):
    from xfastertransformer_b200.ops import native_linear
    monkeypatch.setattr(native_linear, "step_columns", lambda *a: columns)
    M.gated_linear(_dev(), torch.bfloat16, 1.5e-2, 2, 100, 200, 16, 16.0, (40, 9), (1, 3))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("sizes", [(4000,), (1,), (2,), (1, 40, 3, 17)])
@pytest.mark.parametrize("hq,hkv,d,padded,taps", [(3, 1, 20, 64, 3), (6, 2, 128, 128, 4), (2, 2, 96, 128, 2), (1, 1, 264, 264, 7), (4, 1, 36, 64, 1),
                                                  (2, 1, 160, 256, 8), (3, 3, 21, 64, 5), (2, 1, 64, 64, 0)])
def test_head_prep(dtype, tol, hq, hkv, d, padded, taps, sizes):
    rot = {"dims": d // 4 * 2, "base": 3000.0, "scaling": dict(factor=6.0, low=1.0, high=4.0, original=50)}
    padded = d if dtype == torch.float32 else padded
    lengths = (30, 9, 1) if max(sizes) < 3 else (500, 33, 1, 6)
    M.head_prep(_dev(), dtype, tol, hq, hkv, d, padded, taps, lengths, sizes, rot)
    M.head_prep(_dev(), dtype, tol, hq, hkv, d, padded, taps, lengths[1:], sizes, norm=False)


def test_head_prep_long():
    """Runs of tokens per warp that cross from one sequence into the next."""
    M.head_prep(_dev(), torch.bfloat16, 1e-2, 2, 1, 64, 64, 4, (1500, 3, 500, 1, 99), (4000,), {"dims": 64, "base": 1e4})


@pytest.mark.parametrize("H", [72, 100, 256, 1021, 2048, 5120])
def test_residual_extras(H):
    M.residual_extras(_dev(), H, torch.bfloat16, 4e-6)
    M.residual_extras(_dev(), H, torch.float32, 4e-6)


@pytest.mark.parametrize("T", [1, 16, 40, 100, 300, 2000])
@pytest.mark.parametrize("K,N", [(96, 8), (256, 24), (2048, 128), (2048, 256)])
def test_linear_times(T, K, N):
    """The factor in the epilogue of every bf16 product kernel: weight stream, tiles, token-major; and in 32 bits."""
    M.linear_times(_dev(), torch.bfloat16, 8e-3, T, K, N)
    M.linear_times(_dev(), torch.float32, 1e-5, T, K, N)


@pytest.mark.parametrize("E,top,groups", [(12, 3, (4, 2)), (8, 4, (2, 1)), (6, 2, (6, 3)), (9, 9, None), (128, 8, (8, 4)), (62, 5, (31, 7))])
def test_grouped_route(E, top, groups):
    M.grouped_route(_dev(), E, top, groups)


@pytest.mark.parametrize("T,E,top,ff,groups", [(9, 6, 2, 24, (3, 2)), (1, 4, 4, 8, None), (300, 32, 3, 64, (4, 2)), (200, 2, 1, 136, None)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_gated_experts(dtype, tol, T, E, top, ff, groups):
    M.gated_experts(_dev(), dtype, tol, T, E, top, ff, groups=groups)


# ------------------------------------------------------------------------------------------ Dagezen's mechanisms
@KINDS
@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 40, 3, 17), (64, 200, 16, 65)])
@pytest.mark.parametrize("H,d,rank", [(3, 12, 5), (2, 128, 16), (2, 64, 33), (2, 72, 24)])
def test_time_mix(dtype, tol, H, d, rank, sizes):
    n = 70 if max(sizes) < 3 else 300
    M.time_mix(_dev(), dtype, tol, H, d, rank, (n, 33, 1, 130, 6), sizes)


@KINDS
@pytest.mark.parametrize("H,d,rank", [(1, 200, 16), (1, 256, 9), (1, 300, 9), (2, 33, 7), (1, 8, 1), (5, 128, 48)])
def test_time_mix_sizes(dtype, tol, H, d, rank):
    M.time_mix(_dev(), dtype, tol, H, d, rank, (100, 20, 3), (1000,))
    M.time_mix(_dev(), dtype, tol, H, d, rank, (20, 3), (1, 2))


@KINDS
@pytest.mark.parametrize("around,spread", [(-5.0, 0.5), (0.0, 2.0), (2.0, 1.0), (4.0, 3.0), (-12.0, 0.1)])
def test_time_mix_decays(dtype, tol, around, spread):
    """Decays from none to all within a token: chunks in one piece, in pieces, and pieces from differences."""
    M.time_mix(_dev(), dtype, tol, 2, 64, 16, (200, 65, 17), (1000,), around, spread)
    M.time_mix(_dev(), dtype, tol, 1, 136, 16, (90,), (1000,), around, spread)


@pytest.mark.parametrize("H,d", [(2, 64), (1, 128), (1, 136)])
def test_time_mix_segments(H, d):
    M.time_mix(_dev(), torch.bfloat16, 1.5e-2, H, d, 16, (1500, 70, 1130, 33, 3), (2000,), -4.0, 0.5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 5, 3)])
def test_token_shift(dtype, sizes):
    M.token_shift(_dev(), dtype, (300, 9, 1, 2), sizes)
    M.token_shift(_dev(), dtype, (30, 9, 1, 2), sizes, 1048, 3)


STATES = pytest.mark.parametrize("dtype,tol", [(torch.float32, 4e-5), (torch.bfloat16, 2e-2)])


@STATES
@pytest.mark.parametrize("sizes", [(1000,), (1,), (2,), (1, 40, 3, 17), (64, 200, 16, 65)])
@pytest.mark.parametrize("H,P,N,G,parts,taps", [(4, 12, 20, 2, 3, 3), (8, 64, 128, 1, 1, 4), (6, 32, 64, 3, 2, 2)])
def test_state_space(dtype, tol, H, P, N, G, parts, taps, sizes):
    """Token by token, in chunks, and both in one batch."""
    n = 70 if max(sizes) < 3 else 300
    M.state_space(_dev(), dtype, tol, H, P, N, G, parts, taps, (n, 33, 1, 130, 6), sizes)


@STATES
@pytest.mark.parametrize("H,P,N,G,parts,taps", [(1, 200, 256, 1, 1, 8), (2, 136, 300, 2, 4, 5), (3, 21, 33, 1, 3, 1), (2, 128, 96, 2, 1, 4),
                                                (2, 72, 200, 1, 6, 7), (64, 64, 16, 8, 1, 4), (80, 64, 16, 8, 1, 4), (72, 128, 8, 1, 1, 2),
                                                (33, 512, 8, 1, 1, 1)])
def test_state_space_sizes(dtype, tol, H, P, N, G, parts, taps):
    """Columns over several CTAs, sizes without a chunk instance, odd sizes, norm parts that cut through heads."""
    M.state_space(_dev(), dtype, tol, H, P, N, G, parts, taps, (100, 20, 3), (1000,))
    M.state_space(_dev(), dtype, tol, H, P, N, G, parts, taps, (20, 3), (1, 2))


@STATES
@pytest.mark.parametrize("dt,rate", [(-6.0, -2.0), (2.0, 2.0), (0.0, 4.0), (-3.0, 0.0)])
def test_state_space_decays(dtype, tol, dt, rate):
    M.state_space(_dev(), dtype, tol, 4, 64, 64, 1, 1, 4, (200, 65, 17), (1000,), dt, rate)


def test_state_space_long():
    """Runs of tokens per thread of the convolution that cross from one sequence into the next; many chunks."""
    M.state_space(_dev(), torch.bfloat16, 2e-2, 2, 64, 64, 1, 1, 4, (900, 3, 500, 1, 99), (4000,), -3.0)
    M.state_space(_dev(), torch.bfloat16, 2e-2, 4, 16, 64, 1, 1, 3, (4101, 2, 4095), (9000,), -3.0)


TALK = [(6, 3, 20, 64), (16, 4, 128, 128), (4, 4, 64, 64), (1, 1, 64, 64), (3, 1, 100, 128), (32, 8, 128, 128), (24, 2, 64, 64), (13, 13, 64, 64)]


@pytest.mark.parametrize("window", [40, 64, 1, 129, 0])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("H,G,d,padded", TALK)
def test_talking_edges(H, G, d, padded, decode, window):
    """The prompt kernel (units of one head and of two, several blocks of queries) and the decode kernels."""
    M.talking_edges(_dev(), torch.bfloat16, 1.5e-2, H, G, d, padded, window, decode)


@pytest.mark.parametrize("H,G,d,padded", TALK + [(20, 20, 64, 64), (40, 8, 64, 64), (4, 2, 200, 256), (2, 1, 264, 264), (18, 1, 64, 64)])
def test_talking_sizes(H, G, d, padded):
    """Also sizes that only the plain kernel has, portions of a few tokens, and portions beside single tokens."""
    for decode in (False, True):
        M.talking_scores(_dev(), torch.bfloat16, 1.5e-2, H, G, d, padded, 70, decode)
    M.talking_scores(_dev(), torch.bfloat16, 1.5e-2, H, G, d, padded, 70, False, start=148)
    M.talking_scores(_dev(), torch.bfloat16, 1.5e-2, H, G, d, padded, 70, False, extra=(1, 17, 1, 2))
    M.talking_prep(_dev(), torch.bfloat16, 1e-2, H, G, d, padded)


@pytest.mark.parametrize("window", [40, 1, 0])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 8e-3)])
def test_talking_plain_kernel(monkeypatch, dtype, tol, decode, window):
    from xfastertransformer_b200.utils.flags import Env
    monkeypatch.setenv("XFT_TALKING_TC", "0")
    Env.get().reload()
    M.talking_edges(_dev(), dtype, tol, 6, 3, 20, 20 if dtype == torch.float32 else 64, window, decode)
    M.talking_scores(_dev(), dtype, tol, 5, 1, 33, 33, window, decode)
    M.talking_prep(_dev(), dtype, tol, 5, 1, 33, 33)


@pytest.mark.parametrize("decode", [False, True])
def test_talking_far_keys(decode):
    """A key thousands of positions back, just inside and just outside a wide window; decode steps split over many ranges."""
    M.talking_edges(_dev(), torch.bfloat16, 1.5e-2, 16, 4, 128, 128, 1900, decode, T=2100, start=2050)
    M.talking_scores(_dev(), torch.bfloat16, 1.5e-2, 32, 8, 128, 128, 1000, decode, T=1300, start=1240)


@FORMS
@pytest.mark.parametrize("sizes", [dict(), dict(H=2, d=208, rd=80, R=520, dv=144), dict(H=33, d=64, rd=64, R=512, dv=64), dict(H=4, d=16, rd=2, R=12, dv=8)])
def test_latent_sinks(monkeypatch, form, sizes):
    decode, extra = _form(monkeypatch, form)
    M.latent_sinks(_dev(), torch.bfloat16, 1.5e-2, decode, extra=extra, **sizes)


def test_latent_sinks_long_context(monkeypatch):
    """Contexts split over the CTAs of a cluster and over clusters: the sink counts in one of them."""
    for form in ("decode", "portion"):
        decode, _ = _form(monkeypatch, form)
        M.latent_sinks(_dev(), torch.bfloat16, 2e-2, decode, T=2500, H=3, start=2495)


@pytest.mark.parametrize("decode", [False, True])
def test_latent_sinks_fp32(decode):
    M.latent_sinks(_dev(), torch.float32, 1e-5, decode)


@pytest.mark.parametrize("H", [72, 100, 256, 1021, 2048, 5120, 9000])
def test_sum_norm(H):
    M.sum_norm(_dev(), H, torch.bfloat16, 4e-6)
    M.sum_norm(_dev(), H, torch.float32, 4e-6)
    M.sum_norm(_dev(), H, torch.bfloat16, 4e-6, T=400)


@pytest.mark.parametrize("T", [1, 16, 40, 100, 300, 2000])
@pytest.mark.parametrize("K,N", [(96, 8), (256, 24), (2048, 128), (2048, 256)])
def test_clamped_gate_and_activations(T, K, N):
    """The epilogues of every product kernel: weight stream, tiles, token-major; and in 32 bits."""
    M.clamped_gate(_dev(), torch.bfloat16, 8e-3, T, K, N, 0.7)
    M.clamped_gate(_dev(), torch.float32, 1e-5, T, K, N, 7.0)
    M.activations(_dev(), torch.bfloat16, 8e-3, T, K, N)
    M.activations(_dev(), torch.float32, 1e-5, T, K, N)
    M.linear_parts(_dev(), torch.bfloat16, 8e-3, T, K, N)
    M.linear_parts(_dev(), torch.float32, 1e-5, T, K, N)


@pytest.mark.parametrize("T,E,top,ff", [(9, 6, 2, 24), (1, 7, 7, 8), (300, 32, 3, 64), (200, 1, 1, 136)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_chosen_experts(dtype, tol, T, E, top, ff):
    M.chosen_experts(_dev(), dtype, tol, T, E, top, ff)


# ------------------------------------------------------------------------------------------ whole models
BOTH = pytest.mark.parametrize("dtype", ["fp32", "bf16"])


@BOTH
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_whole_prompt(cases, name, dtype):
    C.whole_prompt(cases(name), dtype, 140)


@BOTH
@pytest.mark.parametrize("name", ["unequal", "heads128", "latent", "latent128", "recurrent", "recurrent128", "recurrent_bare"] + C.MIXED_HEADS)
def test_first_tokens(cases, name, dtype):
    C.first_tokens(cases(name), dtype)


@BOTH
@pytest.mark.parametrize("name,start", [("unequal", 1), ("heads128", 40), ("padded", 70), ("shared", 1), ("bare", 100),
                                        ("latent", 1), ("latent128", 40), ("latent_bare", 30), ("latent_large", 100),
                                        ("recurrent", 1), ("recurrent128", 40), ("recurrent_bare", 30), ("recurrent_fast", 1),
                                        ("recurrent_large", 100), ("mixed_heads", 1), ("mixed_heads128", 40),
                                        ("mixed_heads_bare", 30), ("mixed_heads_large", 100)])
def test_token_by_token(cases, name, start, dtype):
    C.token_by_token(cases(name), dtype, 140, start)


@BOTH
@pytest.mark.parametrize("sizes", [(2,), (3, 64, 1), (17, 29)])
@pytest.mark.parametrize("name", ["unequal", "heads128", "latent", "latent128", "recurrent", "recurrent128", "recurrent_fast", "mixed_heads",
                                  "mixed_heads128", "mixed_heads_large"])
def test_portions(cases, name, sizes, dtype):
    C.portions(cases(name), dtype, 140, sizes)


@BOTH
@pytest.mark.parametrize("name", ["unequal", "heads128", "shared", "large_heads"] + C.LATENT + C.RECURRENT + C.MIXED_HEADS)
def test_mixed_batches_reuse_pages(cases, name, dtype):
    assert C.mixed_batches(cases(name), dtype) > 8


@BOTH
@pytest.mark.parametrize("name", ["unequal", "heads128", "latent", "recurrent", "mixed_heads"])
def test_rows_and_order(cases, name, dtype):
    C.rows_and_order(cases(name), dtype)


@BOTH
@pytest.mark.parametrize("name", ["unequal", "heads128", "padded", "latent", "latent128", "recurrent", "recurrent128", "mixed_heads", "mixed_heads128"])
def test_greedy_generation(cases, name, dtype):
    """generate(): the captured decode step (CUDA graph) included."""
    C.greedy(cases(name), dtype, 20, 130)


@pytest.mark.parametrize("name", ["heads128", "latent128", "recurrent128", "mixed_heads128"])
def test_graph_and_eager_steps_agree(cases, monkeypatch, name):
    c = cases(name)
    a = C.greedy(c, "bf16", 30, 60)
    monkeypatch.setenv("XFT_CUDA_GRAPH", "0")
    from xfastertransformer_b200.utils.flags import Env
    Env.get().reload()
    assert C.greedy(c, "bf16", 30, 60) == a


@pytest.mark.parametrize("dtype,kv", [("int8", "bf16"), ("bf16", "int8")])
def test_quantised_weights_and_cache(tmp_path, dtype, kv):
    cfg = O.config([O.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, ff=128, size=30),
                    O.attention_layer(heads=4, kv_heads=2, dim=64, vdim=64, ff=128, size=50, kv_from=0)], width=128, vocab=256)
    W = O.random_weights(cfg)
    p = O.write_checkpoint(str(tmp_path / "q"), cfg, W)
    toks = [(7 * i) % 256 for i in range(90)]
    want = O.forward(cfg, W, toks)
    m = xft.AutoModel.from_pretrained(p, dtype=dtype, kv_cache_dtype=kv)
    assert float((m([toks])[0].double().cpu() - want).pow(2).mean().sqrt() / want.std()) < 0.1
    assert m.generate(torch.tensor([toks]), max_length=100).shape == (1, 100)


def test_long_context_and_table_growth(tmp_path):
    """A prompt past the first rotary table, and generation across its end."""
    cfg = O.config([O.attention_layer(heads=2, kv_heads=1, dim=128, vdim=128, size=300, keep=3, rot_dims=32, ff=64)], width=64,
                   vocab=90)
    W = O.random_weights(cfg)
    p = O.write_checkpoint(str(tmp_path / "long"), cfg, W)
    toks = [(11 * i * i + i) % 90 for i in range(2300)]
    m = xft.AutoModel.from_pretrained(p, dtype="bf16")
    sid = m.set_input_cb([toks], max_length=2400, rows=[[0, 299, 2047, 2048, 2299]])
    got = m.forward_cb()
    m.free_seqs(sid)
    C.check(got, O.forward(cfg, W, toks)[[0, 299, 2047, 2048, 2299]], "bf16", "long prompt")
    assert m.generate(torch.tensor([toks[:2040]]), max_length=2060).shape == (1, 2060)

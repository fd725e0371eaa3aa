"""Dagezen beside Botusun (windowed attention whose values are its keys, gated linear attention, experts) at equal sizes: models and
kernel list for bench_layered.py.

Two models per size, with the same width, depth, attention heads, dense feed-forwards and experts (in turn).  "dagezen": state-space
layers, latent attention and attention with mixed heads beside time mixing in turn.  "botusun", the closest other family: attention
(window 1024) and gated linear attention in turn, no side embedding.
"""
import os

from .bench_layered import VOCAB, _time

# width, attention heads of 128, key/value heads, recurrent heads of 128, dense and expert feed-forwards, layers, batch, prompt length
SIZES = {
    "lite": dict(width=2048, heads=16, kv_heads=4, ff=5632, experts=64, top=6, expert_ff=1408, layers=12, batch=16, input_len=2048),
    "mid": dict(width=4096, heads=32, kv_heads=8, ff=11264, experts=64, top=6, expert_ff=2048, layers=9, batch=16, input_len=2048),
}
DIM, WINDOW, STATE, SSM_VDIM, RANK, KV_RANK, ROT = 128, 1024, 128, 64, 16, 512, 64


def _model(kind, s, tmp):
    import xfastertransformer_b200 as xft
    from xfastertransformer_b200.config import ModelConfig
    from xfastertransformer_b200.tools.synthetic import botusun_config, config_only, dagezen_config
    d = os.path.join(tmp, kind)
    kw = {k: s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "layers")}
    if kind == "dagezen":
        c = dagezen_config(vocab=VOCAB, ff=s["ff"], expert_ff=s["expert_ff"], window=WINDOW, **kw)
    else:
        c = botusun_config(vocab=VOCAB, ff=s["expert_ff"], groups=8, keep=4, window=WINDOW, gla_heads=s["heads"], **kw)
        del c["token_side"], c["loop"]
        for i, e in enumerate(c["layers"]):
            if i // 2 % 2 == 0:                              # both kinds of mixer with both kinds of feed-forward
                e["mlp"] = {"kind": "dense", "ff": s["ff"]}
    config_only(d, ModelConfig.from_dict(c))
    return xft.AutoModel.from_pretrained(d, dtype="bf16", kv_cache_dtype="bf16")


def kernels(s, peaks, only=""):
    """Rows of (kernel, design, tokens, microseconds, bound, fraction of the bound)."""
    import torch

    from xfastertransformer_b200 import ops
    from xfastertransformer_b200.models.decoder import Batch
    from xfastertransformer_b200.ops import native as N
    from xfastertransformer_b200.runtime.loader import make_linear
    dev = torch.device("cuda", 0)
    hbm, tf = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6          # bytes and FLOPs per microsecond
    W, H, G, E, K, F, EF, B, L = (s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff", "expert_ff", "batch", "input_len"))
    rows = []

    def add(name, design, T, fns, nbytes, flops):
        if only and only not in name:
            return
        us = _time(fns)
        bound = max(nbytes / hbm, flops / tf)
        rows.append({"kernel": name, "design": design, "rows": T, "us": round(us, 2), "bound_us": round(bound, 2),
                     "fraction": round(bound / us, 3)})

    def copies(nbytes):
        return max(2, min(40, int(3e8 // max(nbytes, 1)) + 1))

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, device=dev) * s).bfloat16()

    def batch(ql, ctx, nb):
        nblk = (ctx + 63) // 64
        b = Batch(ids=None, positions=None, slots=None, cu_q=[ql * j for j in range(nb + 1)], kv_lens=[ctx] * nb,
                  block_table=torch.randperm(nb * nblk, device=dev).int().view(nb, nblk), is_decode=ql == 1, max_q=ql, max_kv=ctx)
        b.cu_q_dev = torch.arange(0, nb * ql + 1, ql, device=dev, dtype=torch.int32)
        b.kv_lens_dev = torch.full((nb,), ctx, device=dev, dtype=torch.int32)
        b.state_slots = torch.arange(nb, device=dev, dtype=torch.int32)
        return b, nb * nblk

    nb = max(1, 8192 // L)
    one = lambda *n: torch.ones(*n, device=dev)
    # norms and sums
    for T in (8192, B):
        n = copies(T * W * 12)
        xs, ys = [torch.randn(T, W, device=dev) for _ in range(n)], [rnd(T, W) for _ in range(n)]
        w = (one(W), one(W))
        add("norm of the residual sum", "dagezen", T, [lambda x=x, y=y: ops.residual_norm(x, y, w, None, 1e-5, "layer", carry=2.5, post_sum=True,
                                                                                          raw=True) for x, y in zip(xs, ys)], T * W * 12, 0)
        add("residual sum + norm", "botusun", T, [lambda x=x, y=y: ops.residual_norm(x, y, None, (w[0], None), 1e-5, "rms", mult=0.5)
                                                  for x, y in zip(xs, ys)], T * W * 12, 0)
        del xs, ys
    # between projection and recurrence or cache
    SH = 2 * W // SSM_VDIM
    SD = ops.StateDims(SH, STATE, SSM_VDIM, 1, 1, 4, 8)
    TK = ops.TalkingHeads(H, G, DIM, DIM, one(H * DIM), one(G * DIM), one(H) * 0.5, one(H) * 0.1, torch.eye(H, device=dev), 0.7, 8)
    for T, ql, ctx in ((nb * L, L, L), (B, 1, 100)):
        b, _ = batch(ql, ctx, T // ql)
        n_seq = T // ql
        pool = [torch.zeros((T + 63) // 64 + 1, G, 64, DIM, device=dev, dtype=torch.bfloat16) for _ in range(2)]
        slots = torch.arange(T, device=dev, dtype=torch.int32)
        xs = [rnd(T, TK.row) for _ in range(copies(T * TK.row * 2))]
        add("norms over projections + append", "dagezen", T, [lambda x=x: ops.talking_prep(x, TK, 1e-5, *pool, slots) for x in xs],
            T * 2 * (2 * H + 3 * G) * DIM, 0)
        C = (H + G) * DIM
        prep = ops.HeadPrep(H, G, DIM, DIM, torch.rand(4, C, device=dev), one(DIM), one(DIM))
        state = torch.zeros(n_seq, 3, C, device=dev, dtype=torch.bfloat16)
        tab, pos = torch.rand(16384, DIM // 2, device=dev), (torch.arange(T, device=dev) % L).int()
        xs = [rnd(T, C) for _ in range(copies(T * C * 4))]
        add("convolution + norm + rotation + append", "botusun", T, [lambda x=x: ops.head_prep(
            x, prep, 1e-5, pos, tab, DIM // 2, *pool, slots, state, b.state_slots, b.cu_q, b.kv_lens, meta=b) for x in xs],
            T * 2 * (2 * C + G * DIM) + n_seq * 3 * C * (4 if ql == 1 else 2), 0)
        xs, mu, st = [torch.randn(T, W, device=dev) for _ in range(copies(T * W * 14))], torch.rand(5, W, device=dev), torch.zeros(n_seq, W, device=dev)
        add("token shift", "dagezen", T, [lambda x=x: ops.token_shift(x, mu, st, b.state_slots, b.cu_q, b.kv_lens, torch.bfloat16, meta=b)
                                          for x in xs], T * W * 14 + n_seq * W * (8 if ql == 1 else 4), 0)
        del xs
    # recurrences: prompts and decode steps
    sw = ops.StateWeights(torch.rand(4, SD.channels, device=dev), one(SD.channels), one(SH) * -2, one(SH), one(SH), one(SD.inner))
    D = ops.LinearDims(H, DIM, DIM, RANK, 8)
    row = D.up(D.a_at + RANK)
    a2 = rnd(H * DIM, RANK, s=0.25)
    lw = ops.LinearWeights(a2, torch.full((H * DIM,), 2.0, device=dev), 16.0, one(DIM))
    tw = ops.LinearWeights(a2, torch.full((H * DIM,), -2.5, device=dev), 1.0, one(H * DIM), 1.0, one(H, DIM), 1.0)
    for ql, ctx, n_seq in ((L, L, nb), (L, L, B), (8192, 8192, 1), (1, 8192, B), (1, 8192, 128)):
        b, _ = batch(ql, ctx, n_seq)
        T = n_seq * ql
        what = f"{n_seq} decode steps" if ql == 1 else f"{n_seq} prompts of {ql}"
        steps = 2 if ql == 1 else 1
        st = n_seq * SH * STATE * SSM_VDIM * 4
        cs = torch.zeros(n_seq, 3, SD.channels, device=dev, dtype=torch.bfloat16)
        sets = [(rnd(T, SD.row), torch.zeros(n_seq, SH, STATE, SSM_VDIM, device=dev)) for _ in range(copies(T * SD.row * 2 + 2 * st))]
        flops = SH * (64 * (STATE + SSM_VDIM) + 4 * STATE * SSM_VDIM) if ql > 1 else 0
        add("state space (convolution, recurrence, gated norm), " + what, "dagezen", T, [lambda x=x, s_=s_: ops.state_space(
            x, SD, sw, 1e-5, s_, cs, b.state_slots, b.cu_q, b.kv_lens, meta=b) for x, s_ in sets], T * 2 * (SD.row + SD.inner) + st * steps, T * flops)
        del sets
        st = n_seq * H * DIM * DIM * 4
        sets = [(rnd(T, row), torch.zeros(n_seq, H, DIM, DIM, device=dev)) for _ in range(copies(T * row * 2 + 2 * st))]
        flops = H * (64 * 4 * DIM + 4 * DIM * DIM) if ql > 1 else 0
        for name, design, w in (("time mixing, ", "dagezen", tw), ("gated linear attention, ", "botusun", lw)):
            add(name + what, design, T, [lambda x=x, s_=s_, w=w: ops.gated_linear(x, D, w, 1e-5, s_, b.state_slots, b.cu_q, b.kv_lens, meta=b)
                                         for x, s_ in sets], T * 2 * (row + H * DIM) + st * steps, T * flops)
        del sets

    # attention over paged keys; the mix of the heads counts with 2 heads^2 FLOPs per pair
    def attention(ql, ctx, n_seq, window, design):
        b, nblk = batch(ql, ctx, n_seq)
        sets = [(rnd(n_seq * ql, H, DIM), rnd(nblk, G, 64, DIM), rnd(nblk, G, 64, DIM), rnd(n_seq * ql, TK.row)) for _ in
                range(copies(nblk * 64 * G * DIM * 4))]
        seen = n_seq * sum(min(p + 1, window) for p in range(ctx - ql, ctx))
        nbytes = n_seq * (min(ctx, window + ql - 1) * G * DIM * 4 + ql * H * DIM * 4)
        what = f"{n_seq} x {'decode' if ql == 1 else 'prompt'}, context {ctx}, window {window}"
        if design == "dagezen":
            add("attention with mixed heads, " + what, design, n_seq * ql, [lambda q=q, k=k, v=v, x=x: ops.talking_attention(
                q, x, TK, k, v, b.block_table, b.cu_q, b.kv_lens, DIM ** -0.5, window, meta=b) for q, k, v, x in sets],
                nbytes + n_seq * ql * H * DIM * 2, (4.0 * DIM * H + 2.0 * H * H) * seen)
        else:
            sink = torch.zeros(H, device=dev)
            add("attention, " + what, design, n_seq * ql, [lambda q=q, k=k, v=v: ops.paged_attention(
                q, k, v, b.block_table, b.cu_q, b.kv_lens, DIM ** -0.5, group=H // G, meta=b, window=window, sinks=sink) for q, k, v, x in sets],
                nbytes, 4.0 * DIM * H * seen)
    for design in ("dagezen", "botusun"):
        attention(L, L, nb, WINDOW, design)
        attention(1, 8192, B, WINDOW, design)
    # latent attention: with a sink and one gate value per head, and as Vepivik has it
    for ql, ctx, n_seq in ((L, L, nb), (1, 8192, B)):
        b, nblk = batch(ql, ctx, n_seq)
        up = ops.LatentWeights(rnd(H, DIM, KV_RANK, s=0.04), rnd(H, DIM, KV_RANK, s=0.04))
        seen = n_seq * sum(p + 1 for p in range(ctx - ql, ctx))
        for design in ("dagezen", "vepivik"):
            d = ops.LatentDims(H, DIM, ROT, KV_RANK, DIM, True, True, KV_RANK, design == "dagezen", 8)
            sets = [(rnd(n_seq * ql, d.row), rnd(nblk, 1, 64, KV_RANK + ROT)) for _ in range(copies(nblk * 64 * (KV_RANK + ROT) * 2))]
            sink = torch.zeros(H, device=dev) if design == "dagezen" else None
            per = 2.0 * H * (2 * DIM + ROT) if ql > 1 else 2.0 * H * (2 * KV_RANK + ROT)
            proj = 2.0 * H * 2 * DIM * KV_RANK * (n_seq * ctx if ql > 1 else n_seq)
            add(f"latent attention, {n_seq} x {'decode' if ql == 1 else 'prompt'}, context {ctx}", design, n_seq * ql,
                [lambda x=x, c=c: ops.latent_attention(x, d, c, b.block_table, b.cu_q, b.kv_lens, up, (DIM + ROT) ** -0.5, meta=b, sinks=sink)
                 for x, c in sets], n_seq * (ctx * (KV_RANK + ROT) * 2 + ql * H * (3 * DIM + ROT) * 2) + H * 2 * DIM * KV_RANK * 2, per * seen + proj)
            del sets
    torch.cuda.empty_cache()

    # products
    def lin(o, i):
        return make_linear(rnd(o, i, s=i ** -0.5), "bf16")

    def product(name, design, T, n_out, k, fn, out=0):
        if only and only not in name:
            return
        ws = [lin(n_out, k) for _ in range(copies(n_out * k * 2))]
        x = rnd(T, k)
        add(name, design, T, [lambda w=w: fn(x, w) for w in ws], (n_out * k + T * k + T * (out or n_out)) * 2, 2.0 * T * n_out * k)
    for T in (B, 8192):
        bias = torch.zeros(2 * F, device=dev)
        mix, rk = rnd(T, 5 * W), torch.empty(T, row, device=dev, dtype=torch.bfloat16)
        product("gate-up product, clamped, biases", "dagezen", T, 2 * F, W, lambda x, w: ops.linear_gated(x, w, "clamped", bias, 7.0), F)
        product("gate-up product, silu", "botusun", T, 2 * F, W, lambda x, w: ops.linear_gated(x, w), F)
        product("projection of state-space layers", "dagezen", T, SD.row, W, lambda x, w: ops.linear(x, w))
        product("projection of gated linear attention", "botusun", T, row, W, lambda x, w: ops.linear(x, w))
        product("projection of mixed heads", "dagezen", T, TK.row, W, lambda x, w: ops.linear(x, w))
        if not only or "four products" in only:
            ws = [lin(4 * H * DIM, W) for _ in range(copies(4 * H * DIM * W * 2))]
            add("four products of time mixing", "dagezen", T, [lambda w=w: ops.linear_parts(mix[:, :4 * W], w, 4, rk) for w in ws],
                (4 * H * DIM * W + T * 4 * W + T * 4 * H * DIM) * 2, 2.0 * T * 4 * H * DIM * W)
            ws = [lin(RANK, W) for _ in range(8)]
            add("decay's first product", "dagezen", T, [lambda w=w: ops.linear(mix[:, 4 * W:], w, act="tanh", out=rk[:, D.a_at:]) for w in ws],
                (RANK * W + T * W + T * RANK) * 2, 2.0 * T * RANK * W)
        product("output projection of both parts", "dagezen", T, W, 2 * H * DIM, lambda x, w: ops.linear(x, w))
    if not only or only in "experts":
        n_sets = max(1, min(3, int(3e8 // (E * 2 * EF * W * 2)) + 1))
        for design, gated in (("dagezen", False), ("botusun", True)):
            sets = [[(lin((2 if gated else 1) * EF, W), lin(W, EF)) for _ in range(E)] for _ in range(n_sets)]
            router, rb, corr, n_mat = lin(E, W), torch.zeros(E, device=dev), torch.randn(E, device=dev) * 0.01, 3 if gated else 2

            def block(h, ex):
                z = ops.linear(h, router, None if gated else rb, out_dtype=torch.float32)
                r = ops.route(z, "deepseek", K, corr, 8, 4, 1.0, False, "sigmoid") if gated else ops.route(z, "mixtral", K)
                return ops.moe_experts(h, *r, ex, "silu" if gated else "gelu_erf", 0, gated=gated)
            for T in (B, 8192):
                hs = [rnd(T, W) for _ in range(2 if T > B else 1)]
                hit = E * (1 - (1 - K / E) ** T)
                add("experts (router, plan, products, sum)", design, T, [lambda h=h, ex=ex: block(h, ex) for h in hs for ex in sets],
                    n_mat * W * 2 * hit * EF + T * W * 6, 2.0 * T * n_mat * W * K * EF)
            del sets
            torch.cuda.empty_cache()
    N.Workspace.get(dev).check_status()
    return rows

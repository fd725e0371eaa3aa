"""Botusun beside Qwen3-MoE (attention with a norm per head, experts with a gate product) at equal sizes: models and kernel list
for bench_layered.py.

Three models per size.  "botusun": attention (window 1024) and gated linear attention in turn, experts in 8 groups of which 4
are kept, a side embedding of 128 per layer.  "botusun_attention": attention in every layer, no window within the context, one
tap, no side embedding: what is left beside Qwen3-MoE's layer is the 32-bit residual stream, the biases, the sink and the
grouped router.  "qwen3_moe": the closest other family.
"""
import os

from .bench_layered import VOCAB, _time

# width, heads of 128, key/value heads, heads and sizes of gated linear attention, experts, layers, batch, prompt length
SIZES = {
    "lite": dict(width=2048, heads=16, kv_heads=4, gla_heads=16, gla_dim=128, gla_vdim=128, experts=64, top=6, ff=1408, layers=16, batch=16,
                 input_len=2048),
    "mid": dict(width=4096, heads=32, kv_heads=8, gla_heads=32, gla_dim=128, gla_vdim=128, experts=64, top=6, ff=2048, layers=12, batch=16,
                input_len=2048),
    "wide-states": dict(width=6144, heads=48, kv_heads=8, gla_heads=24, gla_dim=256, gla_vdim=256, experts=128, top=8, ff=1536, layers=4,
                        batch=16, input_len=1024),
}
DIM, WINDOW, TAPS, SIDE, RANK = 128, 1024, 4, 128, 16


def _model(kind, s, tmp):
    import xfastertransformer_b200 as xft
    from xfastertransformer_b200.config import ModelConfig
    from xfastertransformer_b200.tools.synthetic import botusun_config, config_only, preset
    d = os.path.join(tmp, kind)
    if kind == "qwen3_moe":
        config_only(d, preset("qwen3-8b", model_type="qwen3_moe", num_layer=s["layers"], hidden_size=s["width"], head_num=s["heads"],
                              kv_head_num=s["kv_heads"], size_per_head=DIM, vocab_size=VOCAB, max_pos_seq_len=8192, inter_size=s["ff"],
                              moe_intermediate_size=s["ff"], sparse_experts=s["experts"], num_experts_per_tok=s["top"],
                              norm_topk_prob=True, do_qk_norm=True))
    else:
        kw = {k: s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff", "layers", "gla_heads", "gla_dim", "gla_vdim")}
        if kind == "botusun_attention":
            kw.update(gla_every=0, window=1 << 20, conv=1, side=0)
        c = botusun_config(vocab=VOCAB, groups=8, keep=4, **kw)
        if kind == "botusun_attention":
            del c["token_side"], c["loop"]
        config_only(d, ModelConfig.from_dict(c))
    return xft.AutoModel.from_pretrained(d, dtype="bf16", kv_cache_dtype="bf16")


def kernels(s, peaks):
    """Rows of (kernel, design, tokens, microseconds, bound, fraction of the bound)."""
    import torch

    from xfastertransformer_b200 import ops
    from xfastertransformer_b200.models.decoder import Batch
    from xfastertransformer_b200.ops import native as N
    from xfastertransformer_b200.ops import reference as R
    from xfastertransformer_b200.runtime.loader import make_linear
    dev = torch.device("cuda", 0)
    hbm, tf = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6          # bytes and FLOPs per microsecond
    W, H, G, E, K, F, B, L = (s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff", "batch", "input_len"))
    GH, GD, GV = s["gla_heads"], s["gla_dim"], s["gla_vdim"]
    rows = []

    def add(name, design, T, us, nbytes, flops):
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
    # norms and sums
    for T in (8192, B):
        xs = [torch.randn(T, W, device=dev) for _ in range(copies(T * W * 12))]
        ys = [torch.randn(T, W, device=dev) for _ in xs]
        w = torch.ones(W, device=dev)
        step = torch.ones(W, device=dev)
        rn = lambda x, y, *a, **kw: ops.residual_norm(x, y, *a, 1e-5, "rms", mult=0.5, **kw)
        add("residual sum + norm (fp32 experts' output)", "botusun", T,
            _time([lambda x=x, y=y: rn(x, y, None, (w, None)) for x, y in zip(xs, ys)]), T * W * 14, 0)
        add("residual sum + copy (fp32 experts' output)", "botusun", T,
            _time([lambda x=x, y=y: rn(x, y, None, None, raw=True) for x, y in zip(xs, ys)]), T * W * 14, 0)
        ys = [y.bfloat16() for y in ys]
        add("side norm + sum + step vector + norm", "botusun", T,
            _time([lambda x=x, y=y: rn(x, y, (w, None), (w, None), add=step) for x, y in zip(xs, ys)]), T * W * 12, 0)
        add("rmsnorm", "qwen3_moe", T, _time([lambda y=y: ops.rmsnorm(y, w, 1e-5) for y in ys]), T * W * 4, 0)
        del xs, ys
    # between projection and cache
    tab = R.rope_table(16384, DIM).to(dev)
    half = tab[:, :DIM // 2].contiguous()
    w = torch.ones(DIM, device=dev)
    for T, ql, ctx in ((nb * L, L, L), (B, 1, 100)):
        b, _ = batch(ql, ctx, T // ql)
        C = (H + G) * DIM
        n = copies(T * C * 4)
        pool = [torch.zeros((T + 63) // 64 + 1, G, 64, DIM, device=dev, dtype=torch.bfloat16) for _ in range(2)]
        pos = (torch.arange(T, device=dev) % L).int()
        slots = torch.arange(T, device=dev, dtype=torch.int32)
        prep = ops.HeadPrep(H, G, DIM, DIM, torch.rand(TAPS, C, device=dev), w, w)
        state = torch.zeros(len(b.kv_lens), TAPS - 1, C, device=dev, dtype=torch.bfloat16)
        xs = [rnd(T, C) for _ in range(n)]
        add("convolution + norm + rotation + append", "botusun", T, _time([lambda x=x: ops.head_prep(
            x, prep, 1e-5, pos, half, DIM // 2, *pool, slots, state, b.state_slots, b.cu_q, b.kv_lens, meta=b) for x in xs]),
            T * 2 * (C + C + G * DIM) + (len(b.kv_lens) * (TAPS - 1) * C * (4 if ql == 1 else 2)), 0)
        xs = [rnd(T, (H + 2 * G) * DIM) for _ in range(n)]
        add("split + norm + rotation + append", "qwen3_moe", T, _time([lambda x=x: ops.qkv_rope_cache(
            x, H, G, DIM, pos, tab, DIM, "half", *pool, None, None, slots, None, w, w, 1e-5) for x in xs]), T * 4 * (H + 2 * G) * DIM, 0)
        del xs
    # gated linear attention: prompts and decode steps, and attention over as long a past
    D = ops.LinearDims(GH, GD, GV, RANK, 8)
    row = D.up(D.a_at + RANK)
    lw = ops.LinearWeights(rnd(GH * GD, RANK, s=0.25), torch.full((GH * GD,), 2.0, device=dev), 16.0, torch.ones(GV, device=dev))
    chunk_flops = 64 * 2 * (GD + GV) + 4 * GD * GV                         # per token and head: scores and their product, state twice
    for ql, ctx, n_seq in ((L, L, nb), (L, L, B), (8192, 8192, 1), (1, 8192, B), (1, 8192, 1), (1, 8192, 128)):
        b, _ = batch(ql, ctx, n_seq)
        T = n_seq * ql
        st = n_seq * GH * GD * GV * 4
        n = copies(T * row * 2 + 2 * st)
        sets = [(rnd(T, row), torch.zeros(n_seq, GH, GD, GV, device=dev)) for _ in range(n)]
        us = _time([lambda x=x, s_=s_: ops.gated_linear(x, D, lw, 1e-5, s_, b.state_slots, b.cu_q, b.kv_lens, meta=b) for x, s_ in sets])
        what = f"{n_seq} decode steps" if ql == 1 else f"{n_seq} prompts of {ql}"
        add("gated linear attention, " + what, "botusun", T, us, T * 2 * (row + GH * GV) + st * (2 if ql == 1 else 1),
            T * GH * (chunk_flops if ql > 1 else 0))
        del sets

    def attention(ql, ctx, n_seq, window, design):
        b, nblk = batch(ql, ctx, n_seq)
        n = copies(nblk * 64 * G * DIM * 4)
        sink = torch.zeros(H, device=dev) if design == "botusun" else None
        sets = [(rnd(n_seq * ql, H, DIM), rnd(nblk, G, 64, DIM), rnd(nblk, G, 64, DIM)) for _ in range(n)]
        us = _time([lambda q=q, k=k, v=v: ops.paged_attention(q, k, v, b.block_table, b.cu_q, b.kv_lens, DIM ** -0.5, group=H // G,
                                                              meta=b, window=window, sinks=sink) for q, k, v in sets])
        kv = min(ctx, window + ql - 1) if window else ctx
        seen = n_seq * sum(min(p + 1, window) if window else p + 1 for p in range(ctx - ql, ctx))
        what = f"attention, {n_seq} x {'decode' if ql == 1 else 'prompt'}, context {ctx}" + (f", window {window}" if window else "")
        add(what, design, n_seq * ql, us, n_seq * (kv * G * DIM * 4 + ql * H * DIM * 4), 4.0 * DIM * H * seen)
    attention(L, L, nb, 0, "qwen3_moe")
    attention(L, L, nb, 0, "botusun")
    attention(L, L, nb, WINDOW // 2, "botusun")
    attention(1, 1088, B, 0, "qwen3_moe")
    attention(1, 8192, B, 0, "qwen3_moe")
    attention(1, 8192, B, WINDOW, "botusun")

    # experts: everything from the normalised state to the fp32 output, and its router
    def lin(o, i):
        return make_linear(rnd(o, i, s=i ** -0.5), "bf16")
    n_sets = max(1, min(3, int(3e8 // (E * 3 * F * W * 2)) + 1))
    sets = [[(lin(2 * F, W), lin(W, F)) for _ in range(E)] for _ in range(n_sets)]
    router, corr = lin(E, W), torch.randn(E, device=dev) * 0.01

    def block(h, ex, grouped):
        z = ops.linear(h, router, out_dtype=torch.float32)
        r = ops.route(z, "deepseek", K, corr, 8, 4, 1.0, False, "sigmoid") if grouped else ops.route(z, "softmax_topk", K)
        return ops.moe_experts(h, *r, ex, "silu", 0)
    for design in ("botusun", "qwen3_moe"):
        for T in (B, 8192):
            hs = [rnd(T, W) for _ in range(2 if T > B else 1)]
            hit = E * (1 - (1 - K / E) ** T)
            us = _time([lambda h=h, ex=ex: block(h, ex, design == "botusun") for h in hs for ex in sets])
            add("experts (router, plan, products, sum)", design, T, us, 3 * W * 2 * hit * F + T * W * 6, 2.0 * T * 3 * W * K * F)
    del sets
    torch.cuda.empty_cache()

    # products
    def product(name, design, T, n_out, k, fn=None):
        ws = [lin(n_out, k) for _ in range(copies(n_out * k * 2))]
        x = rnd(T, k)
        us = _time([lambda w=w: fn(x, w) if fn else ops.linear(x, w) for w in ws])
        add(name, design, T, us, (n_out * k + T * k + T * n_out) * 2, 2.0 * T * n_out * k)
    for T in (B, 8192):
        bias = torch.zeros((H + G) * DIM, device=dev)
        e = rnd(T, 4 * SIDE)
        product("projection (queries, keys) with bias", "botusun", T, (H + G) * DIM, W, lambda x, w: ops.linear(x, w, bias))
        product("projection (queries, keys, values)", "qwen3_moe", T, (H + 2 * G) * DIM, W)
        product("projection of gated linear attention", "botusun", T, row, W)
        product("output projection", "both", T, W, H * DIM)
        product("side gate times embedding", "botusun", T, SIDE, W, lambda x, w: ops.linear(x, w, act="gelu_tanh", times=e[:, SIDE:2 * SIDE]))
        product("product of the gate's size", "both", T, SIDE, W)
        product("side projection", "botusun", T, W, SIDE)
    N.Workspace.get(dev).check_status()
    return rows

"""Vepivik beside DeepSeek (latent attention and experts with a gate product) at equal sizes: models and kernel list for
bench_layered.py.

Three models per size.  "vepivik": attention (window 1024) and latent attention (window 4096) in turn, every second latent
layer reading another's latents.  "vepivik_latent": latent attention in every layer, no window within the context, no sharing,
which is DeepSeek's layer with an output gate and experts without a gate product.  "deepseek": queries straight from the
hidden state, experts in every layer.
"""
import os

from .bench_layered import VOCAB, _time

# width, heads (128 + 64 rotated, values 128), key/value heads of the attention layers, experts, layers, batch, prompt length
SIZES = {
    "lite": dict(width=2048, heads=16, kv_heads=4, experts=64, top=6, ff=1408, shared=2816, layers=16, batch=16, input_len=2048),
    "mid": dict(width=4096, heads=32, kv_heads=8, experts=64, top=6, ff=2048, shared=2048, layers=12, batch=16, input_len=2048),
    "v3-layers": dict(width=7168, heads=128, kv_heads=16, experts=128, top=8, ff=2048, shared=2048, layers=4, batch=16,
                      input_len=1024),
}
RANK, ROT, DIM = 512, 64, 128


def _model(kind, s, tmp):
    import xfastertransformer_b200 as xft
    from xfastertransformer_b200.config import ModelConfig
    from xfastertransformer_b200.tools.synthetic import config_only, preset, vepivik_config
    d = os.path.join(tmp, kind)
    if kind == "deepseek":
        config_only(d, preset("deepseek-v3", num_layer=s["layers"], hidden_size=s["width"], head_num=s["heads"], kv_head_num=s["heads"],
                              vocab_size=VOCAB, max_pos_seq_len=8192, q_lora_rank=0, first_k_dense_replace=0,
                              moe_intermediate_size=s["ff"], dense_experts=s["shared"] // s["ff"], sparse_experts=s["experts"],
                              num_experts_per_tok=s["top"], n_group=1, topk_group=1, topk_method="", scoring_func="softmax",
                              weight_data_type="bf16"))
    else:
        kw = {k: s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff", "shared", "layers")}
        if kind == "vepivik_latent":
            kw.update(latent_only=True, share=False, latent_window=1 << 20)
        config_only(d, ModelConfig.from_dict(vepivik_config(vocab=VOCAB, **kw)))
    return xft.AutoModel.from_pretrained(d, dtype="bf16", kv_cache_dtype="bf16")


def kernels(s, peaks):
    """Rows of (kernel, design, tokens, microseconds, bound, fraction of the bound)."""
    import torch

    from xfastertransformer_b200 import ops
    from xfastertransformer_b200.models.decoder import Batch
    from xfastertransformer_b200.ops import native as N
    from xfastertransformer_b200.ops import native_latent as NL
    from xfastertransformer_b200.ops import reference as R
    from xfastertransformer_b200.runtime.loader import make_linear
    dev = torch.device("cuda", 0)
    hbm, tf = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6          # bytes and FLOPs per microsecond
    W, H, G, E, K, F, B, L = (s[k] for k in ("width", "heads", "kv_heads", "experts", "top", "ff", "batch", "input_len"))
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
        return b, nb * nblk

    def seen(ql, ctx, nb, window):
        return nb * sum(min(p + 1, window) if window else p + 1 for p in range(ctx - ql, ctx))

    # norms
    for T in (8192, B):
        xs = [torch.randn(T, W, device=dev) for _ in range(copies(T * W * 12))]
        ys = [torch.randn(T, W, device=dev) for _ in xs]
        w = torch.ones(W, device=dev)
        add("residual sum + norm (fp32 sublayer output)", "vepivik", T,
            _time([lambda x=x, y=y: ops.residual_norm(x, y, None, (w, None), 1e-5, "rms") for x, y in zip(xs, ys)]), T * W * 14, 0)
        ys = [y.bfloat16() for y in ys]
        add("rmsnorm", "deepseek", T, _time([lambda y=y: ops.rmsnorm(y, w, 1e-5) for y in ys]), T * W * 4, 0)
        del xs, ys
    # latent attention: everything between the packed projection and the output projection
    d = ops.LatentDims(H, DIM, ROT, RANK, DIM, True, True, RANK)
    uk, uv = rnd(H, DIM, RANK, s=RANK ** -0.5), rnd(H, DIM, RANK, s=RANK ** -0.5)
    lw = ops.LatentWeights(uk, uv)
    tab = R.rope_table(16384, ROT).to(dev)

    def latent(ql, ctx, nb, window):
        b, nblk = batch(ql, ctx, nb)
        T, kv = nb * ql, min(ctx, window + ql - 1) if window else ctx
        n = copies(nb * kv * (RANK + ROT) * 2 if ql == 1 else 3e8)
        ps = [rnd(nblk, 1, 64, RANK + ROT) for _ in range(n)]
        xs = [rnd(T, d.row) for _ in range(n)]
        per_head = 2.0 * T * H * RANK * 2 * DIM                            # absorbing, or expanding `kv` rows
        pairs = seen(ql, ctx, nb, window) * H
        what = f"{'decode' if ql == 1 else 'prompt'}, context {ctx}" + (f", window {window}" if window else "")
        mem = nb * kv * (RANK + ROT) * 2 + 4 * H * DIM * RANK + T * H * 2 * (DIM + ROT + 2 * DIM)
        fl = per_head + pairs * 2 * ((2 * RANK + ROT) if ql == 1 else (2 * DIM + ROT))
        add("latent attention, " + what, "vepivik", T, _time([lambda x=x, p=p: ops.latent_attention(
            x, d, p, b.block_table, b.cu_q, b.kv_lens, lw, 0.07, window, meta=b) for x, p in zip(xs, ps)]), mem, fl)
        if ql > 1 and nb * ctx * H <= 1 << 20:                             # the attention kernel of the prompt form alone
            sp = NL._Spans(b.cu_q, b.kv_lens, window, 2, dev)
            o = torch.empty(T, H * DIM, dtype=torch.bfloat16, device=dev)
            flat, kvs = rnd(sp.rows, RANK + ROT), [rnd(sp.rows, 2 * H * DIM) for _ in range(2)]
            add("  attention kernel alone, " + what, "vepivik", T, _time([lambda x=x, k=k: NL.flat_attention(
                x, d, k, flat, sp, 0, H, 0.07, window, o) for x, k in zip(xs, kvs * n)]),
                T * H * 2 * (2 * DIM + ROT + DIM) + nb * kv * H * 4 * DIM, pairs * 2 * (2 * DIM + ROT))
        if window:
            return
        qn, qr = [x[:, :H * DIM].reshape(T, H, DIM) for x in xs], [x[:, H * DIM:d.q_width].reshape(T, H, ROT) for x in xs]
        mem -= T * H * 2 * DIM                                             # no gate
        add("latent attention, " + what, "deepseek", T, _time([lambda a=a, r=r, p=p: ops.mla_attention(
            a, r, p, b.block_table, b.cu_q, b.kv_lens, uk, uv, 0.07, absorbed=ql == 1, meta=b) for a, r, p in zip(qn, qr, ps)]), mem, fl)

    nb = max(1, 8192 // L)
    for window in (0, 1024):
        latent(L, L, nb, window)
    for ctx in (L, 8192):
        latent(1, ctx, B, 0)
    latent(1, 8192, B, 1024)
    for T in (8192, B):
        n = copies(T * d.row * 2)
        xs, pool = [rnd(T, d.row) for _ in range(n)], rnd(256, 1, 64, RANK + ROT)
        pos, w = torch.arange(T, device=dev, dtype=torch.int32), torch.ones(RANK, device=dev)
        mem = T * 2 * (2 * H * ROT + 2 * (RANK + ROT))
        add("rotation + latent norm + append", "vepivik", T, _time([lambda x=x: ops.latent_prep(
            x, d, pos, tab, ROT, w, 1e-5, pool, pos) for x in xs]), mem, 0)
        add("split + rotation + latent norm + append", "deepseek", T, _time([lambda x=x: ops.mla_prep(
            x[:, :d.q_width], x[:, d.q_width:d.gate_at], H, DIM, ROT, RANK, pos, tab, w, 1e-5, pool, pos) for x in xs]),
            mem + T * 4 * H * DIM, 0)
        del xs

    # window attention beside Llama's kernel at as many keys
    def attention(ql, ctx, nb, window, design):
        b, nblk = batch(ql, ctx, nb)
        n = copies(nblk * 64 * G * DIM * 4)
        sets = [(rnd(nb * ql, H, DIM), rnd(nblk, G, 64, DIM), rnd(nblk, G, 64, DIM)) for _ in range(n)]
        us = _time([lambda q=q, k=k, v=v: ops.paged_attention(q, k, v, b.block_table, b.cu_q, b.kv_lens, DIM ** -0.5, group=H // G,
                                                              meta=b, window=window) for q, k, v in sets])
        kv = min(ctx, window + ql - 1) if window else ctx
        what = f"attention, {'decode' if ql == 1 else 'prompt'}, context {ctx}" + (f", window {window}" if window else "")
        add(what, design, nb * ql, us, nb * (kv * G * DIM * 4 + ql * H * DIM * 4), 4.0 * DIM * H * seen(ql, ctx, nb, window))
    attention(L, L, nb, 0, "llama")
    attention(L, L, nb, 1024, "vepivik")
    attention(1, 1088, B, 0, "llama")
    attention(1, 8192, B, 1024, "vepivik")

    # experts: everything from the normalised state to the fp32 output, and its router
    def lin(o, i):
        return make_linear(rnd(o, i, s=i ** -0.5), "bf16")
    n_sets = max(1, min(3, int(3e8 // (E * 2 * F * W * 2)) + 1))
    for design, gated in (("vepivik", False), ("deepseek", True)):
        act = "silu" if gated else "relu2"
        mats = 3 if gated else 2
        sets = [([(lin((mats - 1) * F, W), lin(W, F)) for _ in range(E)], (lin((mats - 1) * s["shared"], W), lin(W, s["shared"])))
                for _ in range(n_sets)]
        router = lin(E, W)

        def block(h, ex, sh):
            idx, w = ops.route(ops.linear(h, router, out_dtype=torch.float32), "deepseek", K, norm_topk=True, scoring="softmax")
            if gated:
                out = ops.moe_experts(h, idx, w, ex, act, 0)
                return out + ops.linear(ops.linear_gated(h, sh[0], act), sh[1], out_dtype=torch.float32)
            add_ = ops.linear(ops.linear(h, sh[0], act=act), sh[1], out_dtype=torch.float32)
            return ops.moe_experts(h, idx, w, ex, act, 0, gated=False, add=add_)
        for T in (B, 8192):
            hs = [rnd(T, W) for _ in range(2 if T > B else 1)]
            hit = E * (1 - (1 - K / E) ** T)
            mem = mats * W * 2 * (hit * F + s["shared"]) + T * W * 6
            us = _time([lambda h=h, ex=ex, sh=sh: block(h, ex, sh) for h in hs for ex, sh in sets])
            add("experts (router, plan, products, sum, shared expert)", design, T, us, mem, 2.0 * T * mats * W * (K * F + s["shared"]))
        del sets
        torch.cuda.empty_cache()

    # products
    def product(name, design, T, n_out, k):
        ws = [lin(n_out, k) for _ in range(copies(n_out * k * 2))]
        x = rnd(T, k)
        add(name, design, T, _time([lambda w=w: ops.linear(x, w) for w in ws]), (n_out * k + T * k + T * n_out) * 2, 2.0 * T * n_out * k)
    for T in (B, 8192):
        product("packed projection (queries, latent, gate)", "vepivik", T, d.row, W)
        product("packed projection (queries, latent)", "deepseek", T, d.gate_at, W)
        product("output projection", "both", T, W, H * DIM)
    N.Workspace.get(dev).check_status()
    return rows

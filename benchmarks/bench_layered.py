"""Prefill and decode of a layered design beside the closest other family at equal sizes and depth, and the kernels of both
one by one: Kafipel beside Llama here, Vepivik beside DeepSeek in bench_vepivik.py, Botusun beside Qwen3-MoE in bench_botusun.py,
Dagezen beside Botusun in bench_dagezen.py.  Run through ``bench.py --design NAME
[--size NAME]``; one GPU, random weights, one JSON line.

Throughput: prompts of `input_len` tokens through `forward()` (prefill and first token), then `steps` decode steps of the
whole batch (the captured step), both timed with CUDA events.  Kernels: each launched over several sets of inputs that
together exceed L2, captured in one CUDA graph, device time per launch; the bound is the larger of algorithmic bytes over
the measured copy bandwidth and FLOPs over the measured bf16 peak (MEASURED_PEAKS.json).
"""
import json
import os
import statistics
import tempfile

# width, query heads, key/value heads (of 128), feed-forward, layers, batch, prompt length
SIZES = {
    "1b": dict(width=2048, heads=16, kv_heads=4, ff=5632, layers=16, batch=16, input_len=2048),
    "8b": dict(width=4096, heads=32, kv_heads=8, ff=14336, layers=32, batch=16, input_len=2048),
    "70b-layers": dict(width=8192, heads=64, kv_heads=8, ff=28672, layers=8, batch=16, input_len=2048),
}
VOCAB = 32000


def _model(kind, s, tmp):
    import xfastertransformer_b200 as xft
    from xfastertransformer_b200.config import ModelConfig
    from xfastertransformer_b200.tools.synthetic import config_only, kafipel_config, preset
    d = os.path.join(tmp, kind)
    if kind == "llama":
        config_only(d, preset("llama-2-7b", num_layer=s["layers"], hidden_size=s["width"], head_num=s["heads"],
                              kv_head_num=s["kv_heads"], size_per_head=128, inter_size=s["ff"], vocab_size=VOCAB,
                              max_pos_seq_len=8192))
    else:
        kw = {k: s[k] for k in ("width", "heads", "kv_heads", "ff", "layers")}
        full = {"window": 1 << 20, "share": False} if kind == "kafipel_full" else {}
        config_only(d, ModelConfig.from_dict(kafipel_config(vocab=VOCAB, **kw, **full)))
    return xft.AutoModel.from_pretrained(d, dtype="bf16", kv_cache_dtype="bf16")


def throughput(model, s, steps, warmup):
    import torch
    from xfastertransformer_b200.ops import native as N
    m = model.model
    B, L = s["batch"], s["input_len"]
    ids = torch.randint(0, VOCAB, (B, L), generator=torch.Generator().manual_seed(1)).pin_memory()
    pre = []
    for _ in range(3):
        model.set_input(ids, max_length=L + warmup + steps + 2, eos_token_id=-2, pad_token_id=0)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        model.forward()
        e1.record()
        torch.cuda.synchronize()
        pre.append(e0.elapsed_time(e1))
    for _ in range(warmup):
        model.forward()
    m.runner.timing, m.runner.step_events = True, []
    for _ in range(steps):
        model.forward()
    torch.cuda.synchronize()
    ms = sum(a.elapsed_time(b) for a, b in m.runner.step_events) / len(m.runner.step_events)
    launches = [g.kernels for g in m.runner.graphs.values()]
    N.Workspace.get(m.ctx.device).check_status()
    model.finalize()
    out = {"prefill_tokens_per_s": round(B * L / min(pre[1:]) * 1e3), "prefill_ms": round(min(pre[1:]), 2),
           "decode_tokens_per_s": round(B / ms * 1e3, 1), "decode_ms": round(ms, 4), "kernels_per_step": launches[-1],
           "weights_gb": round(m.decoder.weight_bytes() / 1e9, 2)}
    return out


# ------------------------------------------------------------------------------------------ kernels
def _time(fns, reps=7):
    """Median device time per launch of closures on distinct data, captured together."""
    import torch
    torch.cuda.synchronize()          # the inputs (lengths and block tables among them) are made on another stream
    st = torch.cuda.Stream()
    with torch.cuda.stream(st):
        for f in fns:
            f()
        st.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=st):
            for f in fns:
                f()
        t = []
        for _ in range(3 + reps):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(st)
            g.replay()
            e1.record(st)
            st.synchronize()
            t.append(e0.elapsed_time(e1) / len(fns) * 1e3)
    from xfastertransformer_b200.ops import native
    native.Workspace.get(torch.device("cuda", 0)).check_status()
    return statistics.median(t[3:])


def kernels(s, peaks):
    """Rows of (kernel, tokens, microseconds, bound, fraction) for the attention and norm kernels of both designs and the
    products they share."""
    import torch
    from xfastertransformer_b200 import ops
    from xfastertransformer_b200.models.decoder import Batch
    from xfastertransformer_b200.ops import native as N
    from xfastertransformer_b200.runtime.loader import make_linear
    dev = torch.device("cuda", 0)
    hbm, tf = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6          # bytes and FLOPs per microsecond
    W, H, G, F, B, L = s["width"], s["heads"], s["kv_heads"], s["ff"], s["batch"], s["input_len"]
    rows = []

    def add(name, design, T, us, nbytes, flops):
        bound = max(nbytes / hbm, flops / tf)
        rows.append({"kernel": name, "design": design, "rows": T, "us": round(us, 2), "bound_us": round(bound, 2),
                     "fraction": round(bound / us, 3)})

    def copies(nbytes):
        return max(2, min(40, int(3e8 // max(nbytes, 1)) + 1))

    # norms: prompt rows and decode rows
    for T in (8192, B):
        n = copies(T * W * 12)
        xs = [torch.randn(T, W, device=dev) for _ in range(n)]
        ys = [torch.randn(T, W, device=dev).bfloat16() for _ in range(n)]
        w = torch.ones(W, device=dev)
        us = _time([lambda x=x, y=y: ops.residual_norm(x, y, (w, None), (w, None), 1e-5) for x, y in zip(xs, ys)])
        add("residual_norm (post norm + sum + pre norm)", "kafipel", T, us, T * W * 12, 0)
        us = _time([lambda y=y: ops.rmsnorm(y, w, 1e-5) for y in ys])
        add("rmsnorm", "llama", T, us, T * W * 4, 0)
        us = _time([lambda y=y: ops.layernorm(y, w, w, 1e-5) for y in ys])
        add("layernorm", "gpt", T, us, T * W * 4, 0)
        del xs, ys
    # attention: (queries per sequence, context), with and without a window
    def attention(ql, ctx, nb, window, ext):
        nblk = (ctx + 63) // 64
        n = copies(nb * nblk * 64 * G * 128 * 4)
        keep = 4
        seen = sum(min(p + 1, window + keep) if window else p + 1 for p in range(ctx - ql, ctx)) * nb
        fns = []
        for i in range(n):
            kc = torch.randn(nb * nblk, G, 64, 128, device=dev).bfloat16()
            vc = torch.randn(nb * nblk, G, 64, 128, device=dev).bfloat16()
            q = torch.randn(nb * ql, H, 128, device=dev).bfloat16()
            bt = torch.randperm(nb * nblk, device=dev).int().view(nb, nblk)
            b = Batch(ids=None, positions=None, slots=None, cu_q=[ql * j for j in range(nb + 1)], kv_lens=[ctx] * nb,
                      block_table=bt, is_decode=ql == 1, max_q=ql, max_kv=ctx)
            b.cu_q_dev = torch.arange(0, nb * ql + 1, ql, device=dev, dtype=torch.int32)
            b.kv_lens_dev = torch.full((nb,), ctx, device=dev, dtype=torch.int32)
            sink = torch.zeros(H, device=dev)
            kw = dict(softcap=50.0, window=window, keep_first=keep if window else 0, sinks=sink) if ext else {}
            fns.append(lambda q=q, kc=kc, vc=vc, b=b, kw=kw: ops.paged_attention(
                q, kc, vc, b.block_table, b.cu_q, b.kv_lens, 128 ** -0.5, group=H // G, meta=b, **kw))
        us = _time(fns)
        kv = min(ctx, window + keep + ql) if window else ctx
        nbytes = nb * (kv * G * 128 * 4 + ql * H * 128 * 4)
        flops = 4.0 * 128 * H * seen
        phase = "prompt" if ql > 1 else "decode"
        what = f"attention, {phase}, context {ctx}" + (f", window {window}" if window else "")
        add(what, "kafipel" if ext else "llama", nb * ql, us, nbytes, flops)
    attention(L, L, 4, 0, False)
    attention(L, L, 4, 0, True)
    attention(L, L, 4, 1024, True)
    attention(1, 1088, B, 0, False)          # as many keys as a decode step sees through the window
    for ctx in (L, 8192):
        attention(1, ctx, B, 0, False)
        attention(1, ctx, B, 0, True)
        attention(1, ctx, B, 1024, True)
    # products of one layer at decode and prompt size; the ones both designs share run the same kernels
    def product(name, design, T, n_out, k, fn):
        nbytes = (n_out * k + T * k + T * n_out) * 2
        n = copies(n_out * k * 2)
        ws = [make_linear(torch.randn(n_out, k, device=dev).bfloat16() * 0.02, "bf16") for _ in range(n)]
        x = torch.randn(T, k, device=dev).bfloat16()
        us = _time([lambda w=w: fn(x, w) for w in ws])
        add(name, design, T, us, nbytes, 2.0 * T * n_out * k)
    for T in (B, 8192):
        res = torch.randn(T, W, device=dev).bfloat16()
        product("o product", "kafipel", T, W, H * 128, lambda x, w: ops.linear(x, w))
        product("o product + residual", "llama", T, W, H * 128, lambda x, w: ops.linear(x, w, None, None, res, 1.0))
        product("gate-up product", "kafipel", T, 2 * F, W, lambda x, w: ops.linear_gated(x, w))
        if T <= 64:
            product("norm + gate-up product", "llama", T, 2 * F, W, lambda x, w: ops.linear_rms(x, w, 1e-5, None, "silu", True))
        product("down product", "kafipel", T, W, F, lambda x, w: ops.linear(x, w))
        product("down product + residual", "llama", T, W, F, lambda x, w: ops.linear(x, w, None, None, res, 1.0))
    # QKV with rotation and cache append; query rows only for a layer that reads another's keys
    from xfastertransformer_b200.ops import reference as R
    tab = R.rope_table(4096, 128).to(dev)
    kc = torch.zeros(64, G, 64, 128, device=dev, dtype=torch.bfloat16)
    vc = torch.zeros_like(kc)
    pos = torch.arange(B, device=dev, dtype=torch.int32)
    for name, design, hkv, eps, rot in (("QKV + rotation + append", "kafipel", G, None, 64), ("Q + rotation", "kafipel", 0, None, 64),
                                        ("norm + QKV + rotation + append", "llama", G, 1e-5, 128)):
        tb = tab[:, :rot].contiguous()
        product(name, design, B, (H + 2 * hkv) * 128, W, lambda x, w: ops.qkv_linear_rope_cache(
            x, w, None, eps, H, hkv, pos, tb, rot, "half", kc, vc, pos))
    N.Workspace.get(dev).check_status()
    return rows


def run(args, clock_sampler, clock_summary, root):
    os.environ["XFT_FAKE_MODEL"] = "2"
    import gc

    import torch

    from . import bench_botusun, bench_dagezen, bench_vepivik
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        pass
    here = {"kafipel": globals(), "vepivik": vars(bench_vepivik), "botusun": vars(bench_botusun),
            "dagezen": vars(bench_dagezen)}[args.design]
    kinds = {"kafipel": ("kafipel", "kafipel_full", "llama"), "vepivik": ("vepivik", "vepivik_latent", "deepseek"),
             "botusun": ("botusun", "botusun_attention", "qwen3_moe"), "dagezen": ("dagezen", "botusun")}[args.design]
    sizes = here["SIZES"]
    if args.size != "all" and args.size not in sizes:
        raise SystemExit(f"--size {args.size}: {args.design} has {sorted(sizes)}")
    out = {"metric": "layered_design_tokens_per_s", "design": args.design, "data": "synthetic token ids; random-init weights",
           "dtype": "bf16", "n_gpus": 1, "steps": args.steps, "warmup": max(args.warmup, 3), "sizes": {}}
    sampler, path = clock_sampler()
    for name in (sizes if args.size == "all" else [args.size]):
        s = sizes[name]
        r = {"config": s}
        for kind in kinds:
            with tempfile.TemporaryDirectory() as tmp:
                model = here["_model"](kind, s, tmp)
                r[kind] = throughput(model, s, args.steps, max(args.warmup, 3))
                del model
                gc.collect()
                torch.cuda.empty_cache()
        r["kernels"] = here["kernels"](s, peaks)
        torch.cuda.empty_cache()
        out["sizes"][name] = r
    out["clocks"] = clock_summary(sampler, path, 0)
    print(json.dumps(out))
    return 0
